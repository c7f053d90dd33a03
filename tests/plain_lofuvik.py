"""A plain, slow restatement of the Lofuvik decoder: whole sequences, no cache, no batch.

One function per mechanism, written from the design's equations with dense tensors and
Python loops (over tokens for the recurrences and the router, over heads for attention).  It
shares nothing with the package: tests compare the engine with it.  ``weights`` maps
checkpoint tensor names to tensors; ``config`` is the dict of config.json.  Everything runs in
the dtype of ``work`` (64-bit by default).
"""

from __future__ import annotations

import math

import torch


# -- small pieces ------------------------------------------------------------------------------
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def log_sigmoid(z):
    return -softplus(-z)


def previous(h: torch.Tensor) -> torch.Tensor:
    """Row t holds the row before it; the first token's is zero."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)


def causal_conv_silu(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, n], the last column weighing the token itself; zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x], dim=0)
    return silu(sum(padded[j : j + x.shape[0]] * taps[:, j] for j in range(n)))


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


# -- rotation ----------------------------------------------------------------------------------
def frequencies(rot: dict) -> tuple:
    """(frequencies f_i, factor of cosine and sine).  f_i = base^(-2i / dims); with ``scaling``
    each is blended with f_i / factor by a ramp over i between two dimensions: the ones that turn
    ``fast`` and ``slow`` times within ``original`` positions."""
    dims, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if scaling is None:
        return plain, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def dimension(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(dimension(scaling["fast"])), 0)
    high = min(math.ceil(dimension(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, n]: element i < dims / 2 is paired with element i + dims / 2."""
    half = rot["dims"] // 2
    f, stretch = frequencies(rot)
    angle = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * torch.tensor(f, dtype=x.dtype)[None, :]
    cos, sin = stretch * torch.cos(angle)[:, None, :], stretch * torch.sin(angle)[:, None, :]
    u, v = x[..., :half], x[..., half : 2 * half]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half :]], dim=-1)


# -- mixers ------------------------------------------------------------------------------------
def wkv(h, w, prefix, m, eps):
    """Time mixing with a state per head whose decay depends on the token, per key channel."""
    length = h.shape[0]
    heads, dim = m["heads"], m["dim"]
    before = previous(h)
    mixed = {s: h + (before - h) * w[f"{prefix}mu.{s}"] for s in "rkvgw"}
    r, k, v = ((mixed[s] @ w[prefix + s].T).view(length, heads, dim) for s in "rkv")
    gate = silu(mixed["g"] @ w[prefix + "g"].T)
    log_rate = torch.tanh(mixed["w"] @ w[prefix + "w1"].T) @ w[prefix + "w2"].T + w[prefix + "w0"]
    decay = torch.exp(-torch.exp(log_rate)).view(length, heads, dim)
    bonus = w[prefix + "u"]
    out = torch.empty(length, heads, dim, dtype=h.dtype)
    for head in range(heads):
        state = torch.zeros(dim, dim, dtype=h.dtype)
        for t in range(length):
            write = torch.outer(k[t, head], v[t, head])
            out[t, head] = (state + bonus[head][:, None] * write).T @ r[t, head]
            state = decay[t, head][:, None] * state + write
    return (rms(out, eps).reshape(length, heads * dim) * w[prefix + "norm"] * gate) @ w[prefix + "o"].T


def delta(h, w, prefix, m, eps):
    """Gated delta rule: the state is decayed, then corrected towards the value of the key."""
    length = h.shape[0]
    heads, kv_heads, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv_silu(h @ w[prefix + s].T, w[f"{prefix}{s}.conv"]) for s in "qkv")
    q = unit(q.view(length, kv_heads, dim)) * dim ** -0.5
    k = unit(k.view(length, kv_heads, dim))
    v = v.view(length, heads, vdim)
    beta = sigmoid(h @ w[prefix + "b"].T)
    decay = torch.exp(-torch.exp(w[prefix + "A_log"]) * softplus(h @ w[prefix + "a"].T + w[prefix + "dt_bias"]))
    out = torch.empty(length, heads, vdim, dtype=h.dtype)
    per = heads // kv_heads
    for head in range(heads):
        g = head // per
        state = torch.zeros(dim, vdim, dtype=h.dtype)
        for t in range(length):
            state = decay[t, head] * state
            u = beta[t, head] * (v[t, head] - state.T @ k[t, g])
            state = state + torch.outer(k[t, g], u)
            out[t, head] = state.T @ q[t, g]
    gate = silu(h @ w[prefix + "g"].T).view(length, heads, vdim)
    return (rms(out, eps) * w[prefix + "norm"] * gate).reshape(length, heads * vdim) @ w[prefix + "o"].T


def attention(h, w, prefix, m, eps):
    """The left side: causal grouped-query attention, q and k normalised over the whole projection
    before the rotation, capped scores, a sink per head, an output gate per element."""
    length = h.shape[0]
    heads, kv_heads, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w[prefix + "q"].T, eps) * w[prefix + "q.norm"]).view(length, heads, dim)
    k = (rms(h @ w[prefix + "k"].T, eps) * w[prefix + "k.norm"]).view(length, kv_heads, dim)
    v = (h @ w[prefix + "v"].T).view(length, kv_heads, vdim)
    q, k = rotate(q, m["rot"]), rotate(k, m["rot"])
    seen = torch.tril(torch.ones(length, length, dtype=torch.bool))
    out = torch.empty(length, heads, vdim, dtype=h.dtype)
    cap = m.get("softcap")
    per = heads // kv_heads
    for head in range(heads):
        scores = (q[:, head] @ k[:, head // per].T) * m["scale"]
        if cap is not None:
            scores = cap * torch.tanh(scores / cap)
        sink = w[prefix + "sink"][head]
        masked = scores.masked_fill(~seen, -math.inf)
        top = torch.maximum(masked.max(dim=-1, keepdim=True).values, sink)
        e = torch.exp(masked - top)
        out[:, head] = (e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))) @ v[:, head // per]
    gate = sigmoid(h @ w[prefix + "g"].T)
    return (out.reshape(length, heads * vdim) * gate) @ w[prefix + "o"].T


def matrix_memory(h, w, prefix, m, eps):
    """The right side: an exponentially gated matrix memory with a normaliser, carried relative to
    a running maximum that starts at zero."""
    length = h.shape[0]
    heads, dim, vdim, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[prefix + "q"].T * dim ** -0.5).view(length, heads, dim)
    k = (h @ w[prefix + "k"].T).view(length, heads, dim)
    v = (h @ w[prefix + "v"].T).view(length, heads, vdim)
    log_in = cap * torch.tanh((h @ w[prefix + "i"].T + w[prefix + "i.b"]) / cap)
    log_forget = log_sigmoid(cap * torch.tanh((h @ w[prefix + "f"].T + w[prefix + "f.b"]) / cap))
    out = torch.empty(length, heads, vdim, dtype=h.dtype)
    for head in range(heads):
        state = torch.zeros(dim, vdim, dtype=h.dtype)
        norm = torch.zeros(dim, dtype=h.dtype)
        top = torch.zeros((), dtype=h.dtype)
        for t in range(length):
            i, f = log_in[t, head], log_forget[t, head]
            new_top = torch.maximum(f + top, i)
            keep, write = torch.exp(f + top - new_top), torch.exp(i - new_top)
            state = keep * state + write * torch.outer(k[t, head], v[t, head])
            norm = keep * norm + write * k[t, head]
            top = new_top
            scale = torch.maximum((norm @ q[t, head]).abs(), torch.exp(-top)) + 1e-6
            out[t, head] = (state.T @ q[t, head]) / scale
    gate = sigmoid(h @ w[prefix + "g"].T)
    return (rms(out, eps).reshape(length, heads * vdim) * w[prefix + "norm"] * gate) @ w[prefix + "o"].T


def side_by_side(h, w, prefix, m, eps):
    """Both mixers on the same input; half the sum of their outputs, each normalised."""
    left = attention(h, w, prefix + "left.", m["left"], eps)
    right = matrix_memory(h, w, prefix + "right.", m["right"], eps)
    return 0.5 * (rms(left, eps) * w[prefix + "left.out"] + rms(right, eps) * w[prefix + "right.out"])


MIXERS = {"wkv": wkv, "delta": delta, "parallel": side_by_side}


# -- feed-forward ------------------------------------------------------------------------------
def routed_feed_forward(h, w, prefix, mlp, chosen_out: list | None = None):
    """Per token the experts with the largest router logits, weighted by a softmax over those."""
    logits = h @ w[prefix + "router"].T + w[prefix + "router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(logits.shape[1]), key=lambda e: (-float(logits[t, e]), e))[: mlp["router"]["top"]]
        if chosen_out is not None:
            chosen_out.append(order)
        weight = torch.softmax(logits[t, order], dim=0)
        for share, e in zip(weight, order):
            p = f"{prefix}e{e}."
            out[t] += share * (w[p + "down"] @ (silu(w[p + "gate"] @ h[t]) * (w[p + "up"] @ h[t])))
    return out


# -- the model ---------------------------------------------------------------------------------
def layer_runs(config: dict) -> list:
    """(layer, whether the embedding output joins the stream right before it) in running order."""
    count = len(config["layers"])
    loop = config.get("loop")
    if loop is None:
        return [(i, False) for i in range(count)]
    runs = [(i, False) for i in range(loop["start"])]
    for turn in range(loop["times"]):
        runs += [(i, turn > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], count)]


def forward(config: dict, weights: dict, tokens, work=torch.float64, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  ``layers_out`` collects the residual stream after every layer run."""
    w = {k: (v.to(work) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    start = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = start.clone()
    for index, joins in layer_runs(config):
        layer, pre = config["layers"][index], f"l{index}."
        if joins:
            x = x + start
        h = rms(x, eps) * w[pre + "norm1"]
        update = MIXERS[layer["type"]](h, w, pre + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            update = update + routed_feed_forward(h, w, pre + "mlp.", layer["mlp"])
        x = x + update
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T


# -- tensors, random weights, small configurations ------------------------------------------------
def tensor_shapes(config: dict, rank: int = 10) -> dict:
    """``rank``: of the decay's two matrices, which no key of the configuration gives."""
    width = config["width"]
    shapes = {"embed": (config["vocab"], width), "final.norm": (width,), "head": (config["vocab"], width)}
    for index, layer in enumerate(config["layers"]):
        pre, m = f"l{index}.", layer["mixer"]
        mix = pre + "mix."
        shapes[pre + "norm1"] = (width,)
        if layer["type"] == "wkv":
            size = m["heads"] * m["dim"]
            shapes.update({f"{mix}mu.{s}": (width,) for s in "rkvgw"})
            shapes.update({f"{mix}{s}": (size, width) for s in "rkvg"})
            shapes.update({mix + "w1": (rank, width), mix + "w2": (size, rank), mix + "w0": (size,),
                           mix + "u": (m["heads"], m["dim"]), mix + "norm": (size,), mix + "o": (width, size)})
        elif layer["type"] == "delta":
            qk, v = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for s, rows in (("q", qk), ("k", qk), ("v", v)):
                shapes.update({mix + s: (rows, width), f"{mix}{s}.conv": (rows, m["conv"])})
            shapes.update({mix + "a": (m["heads"], width), mix + "b": (m["heads"], width), mix + "A_log": (m["heads"],),
                           mix + "dt_bias": (m["heads"],), mix + "norm": (m["vdim"],), mix + "g": (v, width),
                           mix + "o": (width, v)})
        else:
            left, right = m["left"], m["right"]
            q, k = left["heads"] * left["dim"], left["kv_heads"] * left["dim"]
            v, o = left["kv_heads"] * left["vdim"], left["heads"] * left["vdim"]
            p = mix + "left."
            shapes.update({p + "q": (q, width), p + "k": (k, width), p + "v": (v, width), p + "q.norm": (q,), p + "k.norm": (k,),
                           p + "sink": (left["heads"],), p + "g": (o, width), p + "o": (width, o), p + "out": (width,)})
            qk, v = right["heads"] * right["dim"], right["heads"] * right["vdim"]
            p = mix + "right."
            shapes.update({p + "q": (qk, width), p + "k": (qk, width), p + "v": (v, width), p + "g": (v, width),
                           p + "i": (right["heads"], width), p + "f": (right["heads"], width), p + "i.b": (right["heads"],),
                           p + "f.b": (right["heads"],), p + "norm": (v,), p + "o": (width, v), p + "out": (width,)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        experts, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        shapes.update({pre + "mlp.router": (experts, width), pre + "mlp.router.b": (experts,)})
        for e in range(experts):
            shapes.update({f"{pre}mlp.e{e}.gate": (ff, width), f"{pre}mlp.e{e}.up": (ff, width),
                           f"{pre}mlp.e{e}.down": (width, ff)})
    return shapes


def random_weights(config: dict, seed: int, dtype=torch.bfloat16, rank: int = 10) -> dict:
    """Seeded weights whose sizes keep activations of order one and whose gates and decays spread
    over their ranges; stored in ``dtype``."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config, rank).items():
        noise = torch.randn(shape, generator=gen)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm", "out"):
            t = 1.0 + 0.2 * noise
        elif ".mu." in name:
            t = torch.sigmoid(1.5 * noise)
        elif last == "w0":
            t = -2.0 + 1.5 * noise
        elif last == "A_log":
            t = -1.0 + 0.7 * noise
        elif name.endswith("f.b"):
            t = 2.0 + 2.0 * noise
        elif last in ("u", "sink", "dt_bias", "b") and len(shape) <= 2 and shape[-1] != config["width"]:
            t = noise
        elif last == "conv":
            t = 0.7 * noise
        elif name == "embed":
            t = noise
        elif last in ("router", "i", "f", "a", "b"):
            t = 2.0 * noise / math.sqrt(shape[-1])
        else:
            t = 1.2 * noise / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out


def routed(experts=6, top=2, ff=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def wkv_layer(heads=3, dim=16, mlp="routed"):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": routed() if mlp == "routed" else mlp}


def delta_layer(heads=4, kv_heads=2, dim=12, vdim=20, conv=3, mlp="routed"):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": routed() if mlp == "routed" else mlp}


def attention_side(heads=4, kv_heads=2, dim=16, vdim=16, rot_dims=12, base=500.0, scaling=(4.0, 40, 6.0, 1.0), scale=None, softcap=9.0):
    rot = {"base": base, "dims": rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    side = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot,
            "scale": scale if scale is not None else 1.3 / math.sqrt(dim)}
    if softcap is not None:
        side["softcap"] = softcap
    return side


def memory_side(heads=3, dim=12, vdim=20, gate_cap=7.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def parallel_layer(left=None, right=None, mlp="routed"):
    return {"type": "parallel", "mixer": {"left": left or attention_side(), "right": right or memory_side()},
            "mlp": routed() if mlp == "routed" else mlp}


def config(layers, width=64, vocab=89, eps=2e-5, loop=None) -> dict:
    out = {"architecture": "Lofuvik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": list(layers)}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


def greedy_generate(cfg: dict, weights: dict, prompt, count: int) -> list:
    ids = list(prompt)
    for _ in range(count):
        ids.append(int(forward(cfg, weights, ids)[-1].argmax()))
    return ids[len(prompt):]
