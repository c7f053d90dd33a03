// What the matrix-state recurrences share (wkv.cu, delta_rule.cu, matrix_memory.cu, retention.cu).
//
// Each of them keeps, per request and head, a 32-bit state S [dk, dv] that every token first
// changes and reads; they differ in the change (the mechanism M below).  Two ways through an
// entry's tokens:
//
// state_walk - one block per (head, entry) walks the tokens in order, from and to the request's
//   state row.  Thread (column v, part s) keeps the rows d = i * ds + s of column v in
//   registers; the ds threads of a column sit side by side in a warp and add their shares in a
//   butterfly.  Tokens come in chunks of 16 whose vectors and scalars are staged in shared memory
//   (exponentials and norms are taken there, side by side, not inside the chain).  The chain of a
//   chunk runs without a block-wide barrier; afterwards a warp per token takes the head's norm and
//   gate and stores the row.  States too wide for one block's registers are walked in stretches
//   of columns one after the other, their rows normalised by state_head_norm afterwards.
//   Decoding and short portions take this path.
// chunk kernels - portions of SR_LONG_FROM tokens or more run in chunks of SR_LONG tokens: what a
//   chunk adds and how it decays what came before is worked out for all chunks side by side, the
//   states are chained (or, where the chain is a product, walked chunk by chunk), and state_out
//   takes the outputs of all chunks side by side as small 32-bit products from shared memory.
//
// Everything is 32-bit; sums of log decays inside a chunk are 64-bit, so that the exponential of
// a difference of two of them keeps its precision however far both have fallen.
#pragma once
#include "common.cuh"

#define SR_CHUNK 16          // tokens staged at a time by the walk
#define SR_LONG 64           // tokens of a chunk of the chunk-parallel form
#define SR_LONG_FROM 96      // tokens from which on an entry takes that form
#define SR_TP (SR_LONG + 4)  // pitch of a transposed tile [channel][token]

struct StateRun {
  float* state;            // [rows, heads, dk, dv]
  int state_rows;
  const int* slots;        // [entries]
  const int* cu_tokens;    // [entries + 1]
  int heads, dk, dv, ds;
  const float* v;          // value of token t, head h, column c: v[t * v_ld + h * dv + c]
  long long v_ld;
  const float* norm_w;     // weight of head h, column c: norm_w[h * norm_stride + c]; null: none
  int norm_stride;
  const float* gate;       // act(gate[t * gate_ld + h * dv + c]) multiplies the normalised output
  long long gate_ld;
  int gate_act;            // 0 silu, 1 sigmoid
  float eps;
  void* out;               // [tokens, heads * dv]
  float* raw;              // walk in stretches of columns: the outputs before the norm
  int long_from;           // above zero: entries of this many tokens or more are left to the chunk kernels
};

__device__ __forceinline__ float sr_gate(float z, int act) {
  const float s = 1.f / (1.f + expf(-z));
  return act == 0 ? z * s : s;
}
__device__ __forceinline__ float sr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// Sum over the ds neighbouring lanes of a column.
__device__ __forceinline__ float sr_column_sum(float x, int ds) {
  for (int o = ds >> 1; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
  return x;
}

// One row of dv values at `o` (shared memory), by a warp: norm, weight, gate, store.
template <typename TO>
__device__ __forceinline__ void sr_store_row(const StateRun& p, const float* o, float scale, int token, int head) {
  const int lane = threadIdx.x & 31;
  float ss = 0.f;
  for (int c = lane; c < p.dv; c += 32) {
    const float x = o[c] * scale;
    ss = fmaf(x, x, ss);
  }
  const float inv = scale / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
  const float* w = p.norm_w == nullptr ? nullptr : p.norm_w + (size_t)head * p.norm_stride;
  const float* g = p.gate + (size_t)token * p.gate_ld + (size_t)head * p.dv;
  TO* dst = (TO*)p.out + ((size_t)token * p.heads + head) * p.dv;
  for (int c = lane; c < p.dv; c += 32) dst[c] = from_float<TO>(o[c] * inv * (w == nullptr ? 1.f : w[c]) * sr_gate(g[c], p.gate_act));
}

// A mechanism M of the walk has
//   VECS, SCALARS, EXTRA   staged vectors over the key channels and scalars per token; whether it
//                          carries one more column (EXTRA 1) whose value is 1 for every token
//   column(p, slot, head, col, &step)  where a column's state lies and how far apart its rows do
//   begin / stage / end    load what it carries beside S, stage nt tokens' vectors [t][VECS][pitch]
//                          and scalars [t][SCALARS], store what it carries
//   step(S, vec, sc, value, s, ds)     one token for one thread; returns the column's output
//   scale(o, sc, dv)       what a token's output row is multiplied by before anything else
template <class M, typename TO, int KPT, int THREADS>
__global__ void __launch_bounds__(THREADS) state_walk_kernel(const M m, const StateRun p, int tile_cols, int* status) {
  extern __shared__ __align__(16) float smem[];
  pdl_trigger();
  pdl_wait();
  const int head = blockIdx.x, entry = blockIdx.y;
  const int first = p.cu_tokens[entry], count = p.cu_tokens[entry + 1] - first;
  if (count <= 0 || (p.long_from > 0 && count >= p.long_from)) return;
  const int slot = p.slots[entry];
  if (slot < 0 || slot >= p.state_rows) {
    if (threadIdx.x == 0) atomicOr(status, FE_STATUS_BAD_PAGE);
    return;
  }
  const int dk = p.dk, dv = p.dv, ds = p.ds, pitch = KPT * ds;
  float* vec = smem;                                  // [SR_CHUNK][VECS][pitch]; rows past dk stay zero
  float* vs = vec + SR_CHUNK * M::VECS * pitch;       // [SR_CHUNK][dv]
  float* os = vs + SR_CHUNK * dv;                     // [SR_CHUNK][dv + EXTRA]
  float* sc = os + SR_CHUNK * (dv + M::EXTRA);        // [SR_CHUNK][SCALARS], then what M carries
  const int tid = threadIdx.x, warp = tid >> 5, warps = blockDim.x >> 5;
  for (int i = tid; i < SR_CHUNK * M::VECS * pitch; i += blockDim.x) vec[i] = 0.f;
  const int v = tid / ds, s = tid - v * ds;
  for (int col0 = 0; col0 < dv; col0 += tile_cols) {
    const int cols = min(tile_cols, dv - col0);
    const bool last_tile = col0 + cols >= dv;
    const bool extra = M::EXTRA != 0 && v == cols;
    const int col = v < cols ? col0 + v : extra ? dv : -1;
    size_t step = 0;
    float* cell = col >= 0 ? m.column(p, slot, head, col, &step) : nullptr;
    float S[KPT];
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
      const int d = i * ds + s;
      S[i] = (col >= 0 && d < dk) ? cell[(size_t)d * step] : 0.f;
    }
    m.begin(p, slot, head, sc + SR_CHUNK * M::SCALARS);
    __syncthreads();
    for (int c0 = 0; c0 < count; c0 += SR_CHUNK) {
      const int nt = min(SR_CHUNK, count - c0);
      m.stage(p, head, first + c0, nt, vec, pitch, sc);
      for (int i = tid; i < nt * cols; i += blockDim.x) {
        const int t = i / cols, c = i - t * cols;
        vs[t * dv + c] = p.v[(size_t)(first + c0 + t) * p.v_ld + (size_t)head * dv + col0 + c];
      }
      __syncthreads();
      for (int t = 0; t < nt; ++t) {
        const float value = v < cols ? vs[t * dv + v] : extra ? 1.f : 0.f;
        const float o = m.template step<KPT>(S, vec + t * M::VECS * pitch, pitch, sc + t * M::SCALARS, value, s, ds);
        if (col >= 0 && s == 0) os[t * (dv + M::EXTRA) + col] = o;
      }
      __syncthreads();
      for (int t = warp; t < nt; t += warps) {
        const float* row = os + t * (dv + M::EXTRA);
        const float scale = m.scale(row, sc + t * M::SCALARS, dv);
        if (p.raw == nullptr) {
          sr_store_row<TO>(p, row, scale, first + c0 + t, head);
        } else {
          float* dst = p.raw + ((size_t)(first + c0 + t) * p.heads + head) * dv;
          for (int c = col0 + (tid & 31); c < col0 + cols; c += 32) dst[c] = row[c] * scale;
        }
      }
      __syncthreads();
    }
    if (col >= 0 && (col < dv || last_tile)) {
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        const int d = i * ds + s;
        if (d < dk) cell[(size_t)d * step] = S[i];
      }
    }
    if (last_tile) m.end(p, slot, head, sc + SR_CHUNK * M::SCALARS);
  }
}

// Norm and gate of outputs the walk left raw: a warp per (token, head).
template <typename TO>
__global__ void __launch_bounds__(128) state_head_norm_kernel(StateRun p, long long rows) {
  pdl_trigger();
  pdl_wait();
  const long long row = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (row >= rows) return;
  const int token = (int)(row / p.heads), head = (int)(row - (long long)token * p.heads);
  sr_store_row<TO>(p, p.raw + row * p.dv, 1.f, token, head);
}

// How the walk's block is laid out: KPT rows of a column per thread, ds threads per column,
// `tile` columns at a time.
struct WalkShape { int kpt, ds, tile, threads; };

static bool walk_shape(int dk, int dv, int extra, WalkShape* w) {
  const int kpts[4] = {4, 8, 16, 32};
  for (int pass = 0; pass < 2; ++pass)
    for (int kpt : kpts) {
      int ds = 1;
      while (ds * kpt < dk) ds <<= 1;
      if (ds > 32) continue;
      const long long threads = (long long)(dv + extra) * ds;
      if (threads > (pass == 0 ? 512 : kpt == 32 ? 640 : 1024)) continue;
      *w = WalkShape{kpt, ds, dv, (int)((threads + 31) / 32 * 32)};
      return true;
    }
  int ds = 1;
  while (ds * 32 < dk) ds <<= 1;
  if (ds > 32) return false;
  const int tile = 512 / ds - extra;
  *w = WalkShape{32, ds, tile, 512};
  return true;
}

// Whether a walk over these sizes leaves raw outputs for state_head_norm.
static bool walk_in_stretches(int dk, int dv, int extra) {
  WalkShape w;
  return walk_shape(dk, dv, extra, &w) && w.tile < dv;
}

template <class M>
static int launch_walk(const M& m, StateRun p, int out_dtype, int entries, int tokens, int* status, cudaStream_t stream) {
  WalkShape w;
  if (!walk_shape(p.dk, p.dv, M::EXTRA, &w)) return FE_ERR_BAD_SHAPE;
  if (w.tile < p.dv) {
    if (p.raw == nullptr) return FE_ERR_BAD_SHAPE;
  } else {
    p.raw = nullptr;
  }
  p.ds = w.ds;
  const size_t smem = sizeof(float) * ((size_t)SR_CHUNK * (M::VECS * w.kpt * w.ds + 2 * p.dv + M::EXTRA + M::SCALARS) + 8);
  if (smem > 200 * 1024) return FE_ERR_TOO_LARGE;
  int rc = FE_ERR_BAD_DTYPE;
#define SR_WALK(TO, KPT, THREADS)                                                                                        \
  do {                                                                                                                   \
    if (smem > 48 * 1024)                                                                                                \
      cudaFuncSetAttribute(state_walk_kernel<M, TO, KPT, THREADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    rc = fe_launch_dependent(state_walk_kernel<M, TO, KPT, THREADS>, dim3(p.heads, entries), dim3(w.threads), smem, stream, \
                             m, p, w.tile, status);                                                                      \
  } while (0)
#define SR_WALK_BY_KPT(TO)                       \
  do {                                           \
    if (w.kpt == 4) SR_WALK(TO, 4, 1024);        \
    else if (w.kpt == 8) SR_WALK(TO, 8, 1024);   \
    else if (w.kpt == 16) SR_WALK(TO, 16, 1024); \
    else SR_WALK(TO, 32, 640);                   \
  } while (0)
  if (out_dtype == FE_DTYPE_F32) SR_WALK_BY_KPT(float);
  else if (out_dtype == FE_DTYPE_BF16) SR_WALK_BY_KPT(bf16);
#undef SR_WALK_BY_KPT
#undef SR_WALK
  if (rc || p.raw == nullptr) return rc;
  const long long rows = (long long)tokens * p.heads;
  const dim3 grid((unsigned)((rows + 3) / 4));
  return out_dtype == FE_DTYPE_F32 ? fe_launch_dependent(state_head_norm_kernel<float>, grid, dim3(128), 0, stream, p, rows)
                                   : fe_launch_dependent(state_head_norm_kernel<bf16>, grid, dim3(128), 0, stream, p, rows);
}

// ---------------------------------------------------------------------------
// chunk-parallel form
// ---------------------------------------------------------------------------

// Chunk c of entry e has a slot of its own: an entry's chunks take as many slots as it has whole
// stretches of SR_LONG tokens and one more, so floor(first / SR_LONG) + e + c never repeats.
__device__ __forceinline__ int sr_slot(int first, int entry, int chunk) { return first / SR_LONG + entry + chunk; }
static inline long long sr_slots(long long tokens, long long entries) { return tokens / SR_LONG + entries + 1; }

struct ChunkAt { int entry_first, first, count, slot, chunks; };

// The tokens of chunk blockIdx.z of entry blockIdx.y; false where there is none.
__device__ __forceinline__ bool sr_locate(const StateRun& p, ChunkAt* at) {
  const int entry = blockIdx.y, chunk = blockIdx.z;
  const int first = p.cu_tokens[entry], count = p.cu_tokens[entry + 1] - first;
  if (count < p.long_from || chunk * SR_LONG >= count) return false;
  at->entry_first = first;
  at->first = first + chunk * SR_LONG;
  at->count = min(SR_LONG, count - chunk * SR_LONG);
  at->slot = sr_slot(first, entry, chunk);
  at->chunks = (count + SR_LONG - 1) / SR_LONG;
  return true;
}

// acc[a][b] += sum_k xt[k * ldx + row + a] * y[k * ldy + col + b]
__device__ __forceinline__ void sr_mm44(float (&acc)[4][4], const float* xt, int ldx, const float* y, int ldy, int depth,
                                        int row, int col) {
#pragma unroll 4
  for (int k = 0; k < depth; ++k) {
    const float4 x = *reinterpret_cast<const float4*>(xt + k * ldx + row);
    const float4 b = *reinterpret_cast<const float4*>(y + k * ldy + col);
    const float xa[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      acc[a][0] = fmaf(xa[a], b.x, acc[a][0]);
      acc[a][1] = fmaf(xa[a], b.y, acc[a][1]);
      acc[a][2] = fmaf(xa[a], b.z, acc[a][2]);
      acc[a][3] = fmaf(xa[a], b.w, acc[a][3]);
    }
  }
}

// Two 32-bit numbers in a 64-bit register pair, for the packed multiply and multiply-add.
__device__ __forceinline__ uint64_t sr_pair(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 sr_unpair(uint64_t v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ uint64_t sr_fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t sr_mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// Copies of 16 or 4 bytes into shared memory that complete in the background.
__device__ __forceinline__ void sr_copy16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void sr_copy4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void sr_copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void sr_copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Rows of 32-bit numbers `ld` apart.
struct Rows {
  const float* base;
  long long ld;
  __device__ __forceinline__ const float* row(int r) const { return base + (size_t)r * ld; }
  __device__ __forceinline__ bool wide(int width) const {
    return (width & 3) == 0 && (ld & 3) == 0 && ((uintptr_t)base & 15) == 0;
  }
};

// The first `width` numbers of `count` rows (tokens), times `mul`, as a transposed tile
// dst[channel * SR_TP + t]; zero past the last row.  A thread's loads are issued four at a time
// before any is stored; neighbouring lanes take neighbouring rows, so that the stores fall into
// different banks.
__device__ __forceinline__ void sr_stage_transposed(float* dst, const Rows& src, int width, int count, float mul = 1.f) {
  const int step = blockDim.x;
  if (src.wide(width)) {
    const int items = SR_LONG * (width >> 2);
    for (int i0 = threadIdx.x; i0 < items; i0 += 4 * step) {
      float4 x[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = i0 + j * step, t = i & (SR_LONG - 1), d = (i / SR_LONG) * 4;
        x[j] = (i < items && t < count) ? *reinterpret_cast<const float4*>(src.row(t) + d) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = i0 + j * step, t = i & (SR_LONG - 1), d = (i / SR_LONG) * 4;
        if (i < items) {
          float* to = dst + d * SR_TP + t;
          to[0] = x[j].x * mul, to[SR_TP] = x[j].y * mul, to[2 * SR_TP] = x[j].z * mul, to[3 * SR_TP] = x[j].w * mul;
        }
      }
    }
    return;
  }
  const int items = SR_LONG * width;
  for (int i0 = threadIdx.x; i0 < items; i0 += 4 * step) {
    float x[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = i0 + j * step, t = i & (SR_LONG - 1), d = i / SR_LONG;
      x[j] = (i < items && t < count) ? src.row(t)[d] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = i0 + j * step;
      if (i < items) dst[(i / SR_LONG) * SR_TP + (i & (SR_LONG - 1))] = x[j] * mul;
    }
  }
}

// Columns c0 .. c0 + 63 of `count` of `rows` rows of `width` numbers as a tile dst[row * 64 + column];
// zero past the last row and the last column.
__device__ __forceinline__ void sr_stage_columns(float* dst, const Rows& src, int rows, int count, int c0, int width) {
  const int step = blockDim.x;
  if (src.wide(width)) {
    const int items = rows * 16;
    for (int i0 = threadIdx.x; i0 < items; i0 += 4 * step) {
      float4 x[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = i0 + j * step, r = i >> 4, c = c0 + (i & 15) * 4;
        x[j] = (r < count && c < width) ? *reinterpret_cast<const float4*>(src.row(r) + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = i0 + j * step;
        if (i < items) reinterpret_cast<float4*>(dst)[i] = x[j];
      }
    }
    return;
  }
  const int items = rows * 64;
  for (int i0 = threadIdx.x; i0 < items; i0 += 4 * step) {
    float x[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = i0 + j * step, r = i >> 6, c = c0 + (i & 63);
      x[j] = (r < count && c < width) ? src.row(r)[c] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = i0 + j * step;
      if (i < items) dst[i] = x[j];
    }
  }
}

// Inclusive running sum / maximum over 64 numbers held by a warp: element lane in `a`, element
// 32 + lane in `b`.
__device__ __forceinline__ void sr_running_sum(double& a, double& b) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double x = __shfl_up_sync(0xffffffffu, a, o), y = __shfl_up_sync(0xffffffffu, b, o);
    if (lane >= o) a += x, b += y;
  }
  b += __shfl_sync(0xffffffffu, a, 31);
}
__device__ __forceinline__ void sr_running_max(double& a, double& b) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double x = __shfl_up_sync(0xffffffffu, a, o), y = __shfl_up_sync(0xffffffffu, b, o);
    if (lane >= o) a = fmax(a, x), b = fmax(b, y);
  }
  b = fmax(b, __shfl_sync(0xffffffffu, a, 31));
}

// state_out: the outputs of one chunk of one head.  A mechanism M has
//   SCORES            whether the chunk's own tokens join through scores (else M's `local` rows do)
//   out_begin(...)    per token: row term rt, column term ct (64-bit; the weight of token j in token
//                     t's output is exp(rt[t] + ct[j])), the factor ea[t] of the start state's
//                     share and (NORMALISER) the floor fl[t]; called by warp 0
//   queries, keys, others, starts, locals   rows of the chunk: its queries (times query_mul()) and keys
//                     per token, what the scores weigh, the state before the chunk per key channel,
//                     what the chunk's own tokens give (without SCORES)
//   NORMALISER        whether rows are divided by max(|sum|, floor_t) + 1e-6 (M's `start_norm`)
// 256 threads: thread (rg, cg) owns rows 4 rg .. and, in pass n, columns 64 n + 4 cg ..
template <class M, typename TO, int NP>
__global__ void __launch_bounds__(256) state_out_kernel(const M m, const StateRun p) {
  extern __shared__ __align__(16) float smem[];
  pdl_trigger();
  pdl_wait();
  ChunkAt at;
  if (!sr_locate(p, &at)) return;
  const int head = blockIdx.x, dk = p.dk, dv = p.dv, tid = threadIdx.x;
  __shared__ double rt[SR_LONG], ct[SR_LONG];
  __shared__ float ea[SR_LONG], fl[SR_LONG], den[SR_LONG];
  __shared__ float part[16][SR_LONG];
  float* qt = smem;                              // [dk][SR_TP]
  float* as = qt + dk * SR_TP;                   // [SR_LONG tokens j][SR_TP tokens t] (SCORES only)
  float* tile = as + (M::SCORES ? SR_LONG * SR_TP : 0);   // keys [dk][SR_TP], then tiles of 64 columns
  const int rg = tid & 15, cg = tid >> 4, row = 4 * rg;
  sr_stage_transposed(qt, m.queries(p, head, at), dk, at.count, m.query_mul());
  if constexpr (M::SCORES) sr_stage_transposed(tile, m.keys(p, head, at), dk, at.count);
  if (tid < 32) m.out_begin(p, head, at, rt, ct, ea, fl);
  __syncthreads();
  if constexpr (M::SCORES) {
    float a[4][4] = {};
    if (4 * cg <= row + 3) sr_mm44(a, qt, SR_TP, tile, SR_TP, dk, row, 4 * cg);
#pragma unroll
    for (int b = 0; b < 4; ++b) {
      const int j = 4 * cg + b;
      float w[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = row + e;
        w[e] = (j <= t && t < at.count) ? a[e][b] * expf((float)(rt[t] + ct[j])) : 0.f;
      }
      store4(as + j * SR_TP + row, w);
    }
    __syncthreads();
    if constexpr (M::NORMALISER) {
      // four threads a token: the sum of its weights and its query against the start normaliser
      const int t = tid >> 2, g = tid & 3;
      const float* n0 = m.start_norm(p, head, at);
      float own = 0.f, old = 0.f;
#pragma unroll 4
      for (int j = g; j < SR_LONG; j += 4) own += as[j * SR_TP + t];
#pragma unroll 4
      for (int d = g; d < dk; d += 4) old = fmaf(qt[d * SR_TP + t], n0[d], old);
      own = sr_column_sum(fmaf(ea[t], old, own), 4);
      if (g == 0) den[t] = 1.f / (fmaxf(fabsf(own), fl[t]) + 1e-6f);
    }
  }
  float acc[NP][4][4];
  float ss[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int n = 0; n < NP; ++n) {
    const int c0 = 64 * n, col = c0 + 4 * cg;
    float own[4][4] = {}, old[4][4] = {};
    if constexpr (M::SCORES) {
      __syncthreads();
      sr_stage_columns(tile, m.others(p, head, at), SR_LONG, at.count, c0, dv);
      __syncthreads();
      sr_mm44(own, as, SR_TP, tile, 64, min(at.count, row + 4), row, 4 * cg);
    }
    __syncthreads();
    sr_stage_columns(tile, m.starts(p, head, at), dk, dk, c0, dv);
    __syncthreads();
    sr_mm44(old, qt, SR_TP, tile, 64, dk, row, 4 * cg);
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      const int t = row + a;
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        float x = fmaf(ea[t], old[a][b], own[a][b]);
        if constexpr (!M::SCORES) x += (t < at.count && col + b < dv) ? m.locals(p, head, at).row(t)[col + b] : 0.f;
        if constexpr (M::NORMALISER) x *= den[t];
        acc[n][a][b] = x;
        ss[a] = fmaf(x, x, ss[a]);
      }
    }
  }
#pragma unroll
  for (int a = 0; a < 4; ++a) part[cg][row + a] = ss[a];
  __syncthreads();
  const float* w = p.norm_w == nullptr ? nullptr : p.norm_w + (size_t)head * p.norm_stride;
  const bool wide = (dv & 3) == 0 && (p.norm_stride & 3) == 0 && (p.gate_ld & 3) == 0 &&
                    (((uintptr_t)p.norm_w | (uintptr_t)p.gate | (uintptr_t)p.out) & 15) == 0;
#pragma unroll
  for (int a = 0; a < 4; ++a) {
    const int t = row + a;
    if (t >= at.count) continue;
    float sum = 0.f;
#pragma unroll
    for (int g = 0; g < 16; ++g) sum += part[g][t];
    const float inv = 1.f / sqrtf(sum / (float)dv + p.eps);
    const float* g = p.gate + (size_t)(at.first + t) * p.gate_ld + (size_t)head * dv;
    TO* dst = (TO*)p.out + ((size_t)(at.first + t) * p.heads + head) * dv;
#pragma unroll
    for (int n = 0; n < NP; ++n) {
      const int c = 64 * n + 4 * cg;
      if (wide) {
        if (c >= dv) continue;
        float wv[4] = {1.f, 1.f, 1.f, 1.f}, gv[4], y[4];
        if (w != nullptr) load4(w + c, wv);
        load4(g + c, gv);
#pragma unroll
        for (int b = 0; b < 4; ++b) y[b] = acc[n][a][b] * inv * wv[b] * sr_gate(gv[b], p.gate_act);
        store4(dst + c, y);
      } else {
#pragma unroll
        for (int b = 0; b < 4; ++b)
          if (c + b < dv) dst[c + b] = from_float<TO>(acc[n][a][b] * inv * (w == nullptr ? 1.f : w[c + b]) * sr_gate(g[c + b], p.gate_act));
      }
    }
  }
}

static size_t state_out_smem(int dk, bool scores) {
  const size_t keys = scores ? (size_t)dk * SR_TP : 0, cols = (size_t)dk * 64;
  size_t tile = keys > cols ? keys : cols;
  if (scores && tile < SR_LONG * 64) tile = SR_LONG * 64;
  return sizeof(float) * ((size_t)dk * SR_TP + (scores ? SR_LONG * SR_TP : 0) + tile);
}

// Sizes the chunk kernels take; others are walked whatever their length.
static bool chunk_takes(int dk, int dv, bool scores) { return dv <= 256 && state_out_smem(dk, scores) <= 200 * 1024; }

template <class M>
static int launch_out(const M& m, const StateRun& p, int out_dtype, int entries, int chunks, cudaStream_t stream) {
  const size_t smem = state_out_smem(p.dk, M::SCORES);
  int rc = FE_ERR_BAD_DTYPE;
#define SR_OUT(TO, NP)                                                                                             \
  do {                                                                                                             \
    if (smem > 30 * 1024)                                                                                          \
      cudaFuncSetAttribute(state_out_kernel<M, TO, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
    rc = fe_launch_dependent(state_out_kernel<M, TO, NP>, dim3(p.heads, entries, chunks), dim3(256), smem, stream, m, p); \
  } while (0)
#define SR_OUT_BY_DV(TO)                     \
  do {                                       \
    if (p.dv <= 64) SR_OUT(TO, 1);           \
    else if (p.dv <= 128) SR_OUT(TO, 2);     \
    else SR_OUT(TO, 4);                      \
  } while (0)
  if (out_dtype == FE_DTYPE_F32) SR_OUT_BY_DV(float);
  else if (out_dtype == FE_DTYPE_BF16) SR_OUT_BY_DV(bf16);
#undef SR_OUT_BY_DV
#undef SR_OUT
  return rc;
}
