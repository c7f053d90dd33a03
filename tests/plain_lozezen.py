"""A plain, slow restatement of the Lozezen decoder: whole sequences, no cache, no batch.

One function per mechanism, written from the design's equations with dense tensors and
Python loops (over tokens for the recurrences, over heads for attention).  It shares nothing with
the package: tests compare the engine with it.  ``weights`` maps checkpoint tensor names to tensors;
``config`` is the dict of config.json.  Everything runs in the dtype of ``work`` (64-bit by default).
"""

from __future__ import annotations

import math

import torch

DECAY_STRENGTH = 8.0          # of the gated linear recurrence


# -- small pieces ------------------------------------------------------------------------------
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_one(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The stored weight is the distance from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z**3)))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, n], the last column weighing the token itself; zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x], dim=0)
    return sum(padded[j : j + x.shape[0]] * taps[:, j] for j in range(n)) + bias


# -- rotation ----------------------------------------------------------------------------------
def angles(length: int, rot: dict, dtype) -> torch.Tensor:
    """[T, dims / 2]: position times base^(-2i / dims), every frequency divided by ``scaling.factor``."""
    scaling = rot.get("scaling")
    divisor = 1.0 if scaling is None else scaling["factor"]
    freq = [rot["base"] ** (-2.0 * i / rot["dims"]) / divisor for i in range(rot["dims"] // 2)]
    return torch.arange(length, dtype=dtype)[:, None] * torch.tensor(freq, dtype=dtype)[None, :]


def rotate_halves(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, n]: element i < dims / 2 is paired with element i + dims / 2."""
    half = rot["dims"] // 2
    angle = angles(x.shape[0], rot, x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half : 2 * half]
    return torch.cat([u * torch.cos(angle) - v * torch.sin(angle), v * torch.cos(angle) + u * torch.sin(angle), x[..., 2 * half :]], dim=-1)


def rotate_neighbours(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, n]: element 2i is paired with element 2i + 1, for the first ``dims`` elements."""
    dims = rot["dims"]
    angle = angles(x.shape[0], rot, x.dtype)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * torch.cos(angle) - v * torch.sin(angle), v * torch.cos(angle) + u * torch.sin(angle)], dim=-1)
    return torch.cat([turned.flatten(-2), x[..., dims:]], dim=-1)


# -- softmax attention -------------------------------------------------------------------------
def window_mask(length: int, size: int) -> torch.Tensor:
    i, j = torch.arange(length)[:, None], torch.arange(length)[None, :]
    return (j <= i) & (i - j < size)


def chunk_mask(length: int, size: int) -> torch.Tensor:
    i, j = torch.arange(length)[:, None], torch.arange(length)[None, :]
    return (j <= i) & (i // size == j // size)


def softmax_heads(q, k, v, seen, scale) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e]: head h reads key/value head floor(h / (H / G))."""
    length, heads = q.shape[:2]
    per = heads // k.shape[1]
    out = torch.empty(length, heads, v.shape[2], dtype=q.dtype)
    for head in range(heads):
        scores = (q[:, head] @ k[:, head // per].T) * scale
        out[:, head] = torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1) @ v[:, head // per]
    return out


def project_heads(h, w, prefix, m):
    length = h.shape[0]
    kv_heads = m.get("kv_heads") or m["heads"]
    q, k, v = (h @ w[prefix + s].T + w[f"{prefix}{s}.b"] for s in "qkv")
    return q.view(length, m["heads"], m["dim"]), k.view(length, kv_heads, m["dim"]), v.view(length, kv_heads, m["vdim"])


def attention(h, w, prefix, m, eps):
    """Sliding window, biases on q, k and v, neighbours rotated."""
    q, k, v = project_heads(h, w, prefix, m)
    q, k = rotate_neighbours(q, m["rot"]), rotate_neighbours(k, m["rot"])
    out = softmax_heads(q, k, v, window_mask(h.shape[0], m["mask"]["size"]), m["scale"])
    return out.flatten(1) @ w[prefix + "o"].T


def chunked_attention(h, w, prefix, m, eps):
    """The left side: q and k normalised head by head, no rotation, keys of the query's own chunk
    only, one gate per head."""
    q, k, v = project_heads(h, w, prefix, m)
    q, k = rms(q, eps) * w[prefix + "q.norm"], rms(k, eps) * w[prefix + "k.norm"]
    out = softmax_heads(q, k, v, chunk_mask(h.shape[0], m["mask"]["size"]), m["scale"])
    return (out * sigmoid(h @ w[prefix + "g"].T)[:, :, None]).flatten(1) @ w[prefix + "o"].T


# -- recurrences -------------------------------------------------------------------------------
def retention(h, w, prefix, m, eps):
    """The right side: linear attention with a fixed decay per head, q and k rotated."""
    length, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = ((h @ w[prefix + s].T).view(length, heads, dim) for s in "qk")
    v = (h @ w[prefix + "v"].T).view(length, heads, vdim)
    q, k = rotate_halves(q, m["rot"]), rotate_halves(k, m["rot"]) * dim**-0.5
    out = torch.empty(length, heads, vdim, dtype=h.dtype)
    for head in range(heads):
        state = torch.zeros(dim, vdim, dtype=h.dtype)
        for t in range(length):
            state = m["decay"][head] * state + torch.outer(k[t, head], v[t, head])
            out[t, head] = state.T @ q[t, head]
    return (rms(out, eps).flatten(1) * silu(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def parallel(h, w, prefix, m, eps):
    left = chunked_attention(h, w, prefix + "left.", m["left"], eps)
    right = retention(h, w, prefix + "right.", m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def rglru(h, w, prefix, m, eps):
    """Two branches; one is a gate, the other goes through a short convolution and a gated linear
    recurrence whose gates read it block by block."""
    length, width, blocks = h.shape[0], m["width"], m["blocks"]
    y = gelu_tanh(h @ w[prefix + "y"].T + w[prefix + "y.b"])
    u = causal_conv(h @ w[prefix + "x"].T + w[prefix + "x.b"], w[prefix + "conv"], w[prefix + "conv.b"])
    parts = u.view(length, blocks, width // blocks)
    gate = lambda s: torch.stack([sigmoid(parts[:, b] @ w[prefix + s][b].T + w[f"{prefix}{s}.b"][b])  # noqa: E731
                                  for b in range(blocks)], dim=1).flatten(1)
    r, i = gate("ra"), gate("ri")
    log_a = -DECAY_STRENGTH * r * softplus(w[prefix + "lam"])
    write = torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    state, states = torch.zeros(width, dtype=h.dtype), []
    for t in range(length):
        state = torch.exp(log_a[t]) * state + write[t]
        states.append(state)
    return (torch.stack(states) * y) @ w[prefix + "o"].T


MIXERS = {"attention": attention, "rglru": rglru, "parallel": parallel}


# -- feed-forward ------------------------------------------------------------------------------
def feed_forward(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


# -- the model ---------------------------------------------------------------------------------
def forward(config: dict, weights: dict, tokens, work=torch.float64, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  ``layers_out`` collects the residual stream after every layer."""
    w = {k: (v.to(work) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    for index, layer in enumerate(config["layers"]):
        pre = f"l{index}."
        update = MIXERS[layer["type"]](norm_around_one(x, w[pre + "norm1"], eps), w, pre + "mix.", layer["mixer"], eps)
        x = x + norm_around_one(update, w[pre + "norm1b"], eps)
        if layer.get("mlp") is not None:
            update = feed_forward(norm_around_one(x, w[pre + "norm2"], eps), w, pre + "mlp.")
            x = x + norm_around_one(update, w[pre + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm_around_one(x, w["final.norm"], eps) @ w["head"].T


# -- tensors, random weights, small configurations ------------------------------------------------
def tensor_shapes(config: dict) -> dict:
    width = config["width"]
    shapes = {"embed": (config["vocab"], width), "final.norm": (width,), "head": (config["vocab"], width)}

    def heads_of(p, m):
        kv_heads = m.get("kv_heads") or m["heads"]
        for s, rows in (("q", m["heads"] * m["dim"]), ("k", kv_heads * m["dim"]), ("v", kv_heads * m["vdim"])):
            shapes.update({p + s: (rows, width), f"{p}{s}.b": (rows,)})
        shapes[p + "o"] = (width, m["heads"] * m["vdim"])

    for index, layer in enumerate(config["layers"]):
        pre, m = f"l{index}.", layer["mixer"]
        mix = pre + "mix."
        shapes.update({pre + "norm1": (width,), pre + "norm1b": (width,)})
        if layer["type"] == "attention":
            heads_of(mix, m)
        elif layer["type"] == "rglru":
            size, blocks = m["width"], m["blocks"]
            part = size // blocks
            for s in "yx":
                shapes.update({mix + s: (size, width), f"{mix}{s}.b": (size,)})
            for s in ("ra", "ri"):
                shapes.update({mix + s: (blocks, part, part), f"{mix}{s}.b": (blocks, part)})
            shapes.update({mix + "conv": (size, m["conv"]), mix + "conv.b": (size,), mix + "lam": (size,), mix + "o": (width, size)})
        else:
            left, right = m["left"], m["right"]
            p = mix + "left."
            heads_of(p, left)
            shapes.update({p + "q.norm": (left["dim"],), p + "k.norm": (left["dim"],), p + "g": (left["heads"], width)})
            p, qk, v = mix + "right.", right["heads"] * right["dim"], right["heads"] * right["vdim"]
            shapes.update({p + "q": (qk, width), p + "k": (qk, width), p + "v": (v, width), p + "g": (v, width), p + "o": (width, v)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            shapes.update({pre + "norm2": (width,), pre + "norm2b": (width,), pre + "mlp.gate": (ff, width),
                           pre + "mlp.up": (ff, width), pre + "mlp.down": (width, ff)})
    return shapes


def random_weights(config: dict, seed: int, dtype=torch.bfloat16) -> dict:
    """Seeded weights whose sizes keep activations of order one and whose decays spread from slow to
    fast; stored in ``dtype``."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        noise = torch.randn(shape, generator=gen)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            t = 0.2 * noise
        elif last == "norm":
            t = 1.0 + 0.2 * noise
        elif last == "lam":
            t = -4.0 + 2.0 * noise
        elif last == "b":
            t = 0.5 * noise
        elif last == "conv":
            t = 0.6 * noise
        elif name == "embed":
            t = noise / config["embedding"]["scale"]
        elif last in ("ra", "ri"):
            t = 1.5 * noise / math.sqrt(shape[-1])
        else:
            t = 1.2 * noise / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def attention_layer(heads=4, kv_heads=2, dim=16, vdim=24, size=20, rot_dims=12, base=300.0, factor=4.0, scale=None, mlp="dense"):
    rot = {"base": base, "dims": rot_dims}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": rot,
             "scale": scale if scale is not None else 1.3 / math.sqrt(dim)}
    if kv_heads is not None:
        mixer["kv_heads"] = kv_heads
    return {"type": "attention", "mixer": mixer, "mlp": dense() if mlp == "dense" else mlp}


def rglru_layer(width=48, blocks=3, conv=3, mlp="dense"):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": dense() if mlp == "dense" else mlp}


def chunk_side(heads=4, kv_heads=2, dim=12, vdim=20, size=18, scale=None):
    side = {"heads": heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale if scale is not None else 1.4 / math.sqrt(dim)}
    if kv_heads is not None:
        side["kv_heads"] = kv_heads
    return side


def retention_side(heads=3, dim=12, vdim=20, rot_dims=8, base=700.0, decay=None):
    decay = decay if decay is not None else [1.0 - 2.0 ** (-2 - h) for h in range(heads)]
    return {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims}, "decay": decay}


def parallel_layer(left=None, right=None, left_scale=0.7, right_scale=1.3, mlp="dense"):
    return {"type": "parallel", "mlp": dense() if mlp == "dense" else mlp,
            "mixer": {"left": left or chunk_side(), "right": right or retention_side(), "left_scale": left_scale, "right_scale": right_scale}}


def config(layers, width=64, vocab=89, eps=2e-5, scale=5.0) -> dict:
    return {"architecture": "Lozezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": list(layers)}


def greedy_generate(cfg: dict, weights: dict, prompt, count: int) -> list:
    ids = list(prompt)
    for _ in range(count):
        ids.append(int(forward(cfg, weights, ids)[-1].argmax()))
    return ids[len(prompt):]
