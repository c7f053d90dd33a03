// The gated delta rule: a state per head that is decayed and then corrected towards each key's value.
//
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//     beta = sigmoid(zb),  g = exp(-exp(A) softplus(za + b)),   per head
//
// q, k and v pass a short causal convolution over time and silu, q and k are made unit vectors per
// head (q times dk^(-1/2)); groups of heads share a q/k head.  A head's o is divided by its root
// mean square, weighted and gated.
//
//   delta_prepare   convolutions, silu, unit vectors, beta and log g of a token; the last taps - 1
//                   rows of the convolution's input stay in the request's state.
//   state_walk      (state_recurrence.cuh) short entries.
//   delta_solve / delta_chain / state_out   long entries in chunks.  With c_t the sum of log g from the
//                   chunk's first token up to t and S the state before the chunk, the u of a chunk solve
//                     u_t + sum_(j < t) L_tj u_j = beta_t (v_t - e^(c_t) S^T k_t),
//                     L_tj = beta_t e^(c_t - c_j) k_t . k_j,
//                   a unit lower triangular system.  delta_solve solves it for all chunks side by side, once
//                   for the right side beta v and once for beta e^c k, so that u = U - W S; delta_chain walks
//                   the chunks with two products each (u, and the state it leads to); then
//                     o_t = e^(c_t) S^T q_t + sum_(j <= t) e^(c_t - c_j) (q_t . k_j) u_j.
#include "state_recurrence.cuh"

// ---------------------------------------------------------------------------
// delta_prepare
// ---------------------------------------------------------------------------
struct DeltaPrepare {
  const float* proj;        // [tokens, ld]: q, k, v from column 0, zb and za at b_off, a_off
  long long ld;
  int b_off, a_off;
  const float* conv;        // [taps, channels]
  int taps;
  float* state;             // [rows, taps - 1, channels], oldest first
  const int *slots, *cu_tokens, *token_entry;
  const float *a_log, *dt_bias;     // [heads]
  int kv_heads, dk, heads, dv;
  float* out;               // [tokens, channels]: q, k unit vectors, v
  float* gates;             // [tokens, heads, 2]: beta, log g
  int n_tokens;
};

#define DP_WARPS 4

// One token's channels of one row - a q, k or v head - by a warp: convolution from `input(j)` (the
// inputs j tokens back), silu, and for q and k the unit vector.  `buf` is the warp's own; a lane reads
// back only what it wrote.  V: neighbouring channels a lane takes at a time.
template <int V> __device__ __forceinline__ void dp_load(const float* p, float* v) { if constexpr (V == 4) load4(p, v); else v[0] = p[0]; }
template <int V> __device__ __forceinline__ void dp_store(float* p, const float* v) { if constexpr (V == 4) store4(p, v); else p[0] = v[0]; }

template <int V, typename F>
__device__ __forceinline__ void delta_prepare_row(const DeltaPrepare& p, int t, int r, float* buf, F input) {
  const int qk = p.kv_heads * p.dk, channels = 2 * qk + p.heads * p.dv, lane = threadIdx.x & 31;
  const bool unit = r < 2 * p.kv_heads;
  const int base = unit ? r * p.dk : 2 * qk + (r - 2 * p.kv_heads) * p.dv, size = unit ? p.dk : p.dv;
  float* out = p.out + (size_t)t * channels + base;
  float ss = 0.f;
  for (int d = lane * V; d < size; d += 32 * V) {
    float y[V], w[V], x[V];
#pragma unroll
    for (int e = 0; e < V; ++e) y[e] = 0.f;
#pragma unroll 4
    for (int j = p.taps - 1; j >= 0; --j) {
      dp_load<V>(p.conv + (size_t)(p.taps - 1 - j) * channels + base + d, w), dp_load<V>(input(j) + base + d, x);
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = fmaf(w[e], x[e], y[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      y[e] = y[e] / (1.f + expf(-y[e]));
      ss = fmaf(y[e], y[e], ss);
    }
    dp_store<V>(unit ? buf + d : out + d, y);
  }
  if (!unit) return;
  const float inv = (r < p.kv_heads ? 1.f / sqrtf((float)p.dk) : 1.f) / sqrtf(warp_sum(ss) + 1e-6f);
  for (int d = lane * V; d < size; d += 32 * V) {
    float y[V];
    dp_load<V>(buf + d, y);
#pragma unroll
    for (int e = 0; e < V; ++e) y[e] *= inv;
    dp_store<V>(out + d, y);
  }
}

__device__ __forceinline__ void delta_prepare_gates(const DeltaPrepare& p, int t) {
  const float* src = p.proj + (size_t)t * p.ld;
  for (int h = threadIdx.x; h < p.heads; h += blockDim.x) {
    float* dst = p.gates + ((size_t)t * p.heads + h) * 2;
    dst[0] = 1.f / (1.f + expf(-src[p.b_off + h]));
    dst[1] = -expf(p.a_log[h]) * sr_softplus(src[p.a_off + h] + p.dt_bias[h]);
  }
}

template <int V>
__global__ void __launch_bounds__(32 * DP_WARPS) delta_prepare_kernel(DeltaPrepare p) {
  extern __shared__ __align__(16) float smem[];      // [DP_WARPS][dk]
  pdl_trigger();
  pdl_wait();
  const int back = p.taps - 1, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int r = blockIdx.y * DP_WARPS + warp, rows = 2 * p.kv_heads + p.heads;
  float* buf = smem + warp * p.dk;
  if ((int)blockIdx.x < p.n_tokens) {
    // a token with all its taps inside the step
    const int t = blockIdx.x;
    if (t - p.cu_tokens[p.token_entry[t]] < back) return;
    if (r < rows) delta_prepare_row<V>(p, t, r, buf, [&](int j) { return p.proj + (size_t)(t - j) * p.ld; });
    if (blockIdx.y == 0) delta_prepare_gates(p, t);
    return;
  }
  // an entry's edge: its first taps - 1 tokens, then the state for the next step
  const int entry = blockIdx.x - p.n_tokens;
  const int first = p.cu_tokens[entry], count = p.cu_tokens[entry + 1] - first, edge = min(count, back);
  if (count <= 0) return;
  if (blockIdx.y == 0)
    for (int i = 0; i < edge; ++i) delta_prepare_gates(p, first + i);
  if (r >= rows) return;
  const int qk = p.kv_heads * p.dk, channels = 2 * qk + p.heads * p.dv;
  float* st = p.state + (size_t)p.slots[entry] * back * channels;
  for (int i = 0; i < edge; ++i)
    delta_prepare_row<V>(p, first + i, r, buf, [&](int j) {
      return j <= i ? p.proj + (size_t)(first + i - j) * p.ld : (const float*)st + (size_t)(back + i - j) * channels;
    });
  // the last taps - 1 rows of (state rows, the step's rows), once the warp has read the old ones; a
  // channel is one lane's here, which reads a state row only before it overwrites it
  __syncwarp();
  const int base = r < 2 * p.kv_heads ? r * p.dk : 2 * qk + (r - 2 * p.kv_heads) * p.dv;
  for (int d = lane; d < (r < 2 * p.kv_heads ? p.dk : p.dv); d += 32)
    for (int k = 0; k < back; ++k) {
      const int at = count + k;
      st[(size_t)k * channels + base + d] =
          at < back ? st[(size_t)at * channels + base + d] : p.proj[(size_t)(first + at - back) * p.ld + base + d];
    }
}

FE_EXPORT int fe_delta_prepare(const float* proj, long long ld, int b_off, int a_off, const float* conv, int taps, float* state,
                               const int* slots, const int* cu_tokens, const int* token_entry, const float* a_log,
                               const float* dt_bias, int kv_heads, int dk, int heads, int dv, float* out, float* gates,
                               int n_tokens, int n_entries, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (taps < 1 || kv_heads < 1 || heads < 1 || dk < 1 || dv < 1 || heads % kv_heads || (taps > 1 && state == nullptr)) return FE_ERR_BAD_SHAPE;
  DeltaPrepare p{proj, ld, b_off, a_off, conv, taps, state, slots, cu_tokens, token_entry, a_log, dt_bias, kv_heads, dk, heads, dv, out, gates, n_tokens};
  const size_t smem = sizeof(float) * (size_t)DP_WARPS * dk;
  const int pieces = (2 * kv_heads + heads + DP_WARPS - 1) / DP_WARPS;
  if (smem > 48 * 1024 || pieces > 65535) return FE_ERR_TOO_LARGE;
  const bool wide = dk % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 &&
                    (((uintptr_t)proj | (uintptr_t)conv | (uintptr_t)state | (uintptr_t)out) & 15) == 0;
  const dim3 grid(n_tokens + (taps > 1 ? n_entries : 0), pieces);
  const int rc = wide ? fe_launch_dependent(delta_prepare_kernel<4>, grid, dim3(32 * DP_WARPS), smem, stream, p)
                      : fe_launch_dependent(delta_prepare_kernel<1>, grid, dim3(32 * DP_WARPS), smem, stream, p);
  return rc ? rc : fe_last_error();
}

// ---------------------------------------------------------------------------
// the recurrence
// ---------------------------------------------------------------------------
struct Delta {
  const float* qkv;         // [tokens, channels]
  long long ld;
  int kv_heads, per;        // q/k heads; heads per q/k head
  const float* gates;       // [tokens, heads, 2]
  // chunk-parallel scratch, per (slot, head)
  float* w;                 // [dk][SR_LONG]: W transposed
  float* u;                 // [SR_LONG][dv]: U, then (chain) u
  float* before;            // [dk, dv]: the state before the chunk
  float* decays;            // [SR_LONG + 4]: e^(c_end - c_t) per token, then e^(c_end)

  static constexpr int VECS = 2, SCALARS = 2, EXTRA = 0;
  static constexpr bool SCORES = true, NORMALISER = false;

  __device__ __forceinline__ const float* q_row(const StateRun& p, int head, int token) const {
    return qkv + (size_t)token * ld + (size_t)(head / per) * p.dk;
  }
  __device__ __forceinline__ const float* k_row(const StateRun& p, int head, int token) const {
    return q_row(p, head, token) + (size_t)kv_heads * p.dk;
  }
  __device__ __forceinline__ float beta(const StateRun& p, int head, int token) const { return gates[((size_t)token * p.heads + head) * 2]; }
  __device__ __forceinline__ float log_decay(const StateRun& p, int head, int token) const { return gates[((size_t)token * p.heads + head) * 2 + 1]; }

  __device__ __forceinline__ float* column(const StateRun& p, int slot, int head, int col, size_t* step) const {
    *step = p.dv;
    return p.state + ((size_t)slot * p.heads + head) * p.dk * p.dv + col;
  }
  __device__ __forceinline__ void begin(const StateRun&, int, int, float*) const {}
  __device__ __forceinline__ void end(const StateRun&, int, int, const float*) const {}
  __device__ __forceinline__ void stage(const StateRun& p, int head, int first, int nt, float* vec, int pitch, float* sc) const {
    for (int i = threadIdx.x; i < nt * p.dk; i += blockDim.x) {
      const int t = i / p.dk, d = i - t * p.dk;
      float* dst = vec + t * VECS * pitch + d;
      dst[0] = q_row(p, head, first + t)[d], dst[pitch] = k_row(p, head, first + t)[d];
    }
    for (int t = threadIdx.x; t < nt; t += blockDim.x) {
      sc[t * SCALARS] = beta(p, head, first + t);
      sc[t * SCALARS + 1] = expf(log_decay(p, head, first + t));
    }
  }
  template <int KPT>
  __device__ __forceinline__ float step(float (&S)[KPT], const float* vec, int pitch, const float* sc, float value, int s, int ds) const {
    const float *qs = vec + s, *ks = qs + pitch;
    const float g = sc[1];
    float have = 0.f;
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
      S[i] *= g;
      have = fmaf(S[i], ks[i * ds], have);
    }
    const float u = sc[0] * (value - sr_column_sum(have, ds));
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
      S[i] = fmaf(ks[i * ds], u, S[i]);
      acc = fmaf(S[i], qs[i * ds], acc);
    }
    return sr_column_sum(acc, ds);
  }
  __device__ __forceinline__ float scale(const float*, const float*, int) const { return 1.f; }

  // -- chunk form --
  // sums of log g up to the chunk's tokens lane and 32 + lane, by one warp (tokens past the end keep
  // the last sum)
  __device__ __forceinline__ void chunk_sums(const StateRun& p, int head, const ChunkAt& at, double* c) const {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int h = 0; h < 2; ++h) c[h] = lane + 32 * h < at.count ? (double)log_decay(p, head, at.first + lane + 32 * h) : 0.0;
    sr_running_sum(c[0], c[1]);
  }
  __device__ __forceinline__ size_t cell(const StateRun& p, const ChunkAt& at, int head) const { return (size_t)at.slot * p.heads + head; }
  __device__ __forceinline__ Rows queries(const StateRun& p, int head, const ChunkAt& at) const { return Rows{q_row(p, head, at.first), ld}; }
  __device__ __forceinline__ float query_mul() const { return 1.f; }
  __device__ __forceinline__ Rows keys(const StateRun& p, int head, const ChunkAt& at) const { return Rows{k_row(p, head, at.first), ld}; }
  __device__ __forceinline__ Rows others(const StateRun& p, int head, const ChunkAt& at) const {
    return Rows{u + cell(p, at, head) * SR_LONG * p.dv, p.dv};
  }
  __device__ __forceinline__ Rows starts(const StateRun& p, int head, const ChunkAt& at) const {
    return Rows{before + cell(p, at, head) * p.dk * p.dv, p.dv};
  }
  __device__ __forceinline__ void out_begin(const StateRun& p, int head, const ChunkAt& at, double* rt, double* ct, float* ea, float*) const {
    double c[2];
    chunk_sums(p, head, at, c);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = (threadIdx.x & 31) + 32 * h;
      rt[t] = c[h];
      ct[t] = -c[h];
      ea[t] = t < at.count ? expf((float)c[h]) : 0.f;
    }
  }
};

// W and U of one chunk of one head: the triangular system solved for the columns of beta e^c k
// and beta v, sixteen rows at a time.  A block of rows first loses what the rows before it give (a
// small product), then a thread per column solves the 16 x 16 triangle in registers and stores the
// result, also for the blocks below.
#define DS_THREADS 256
__global__ void __launch_bounds__(DS_THREADS) delta_solve_kernel(const Delta m, const StateRun p) {
  extern __shared__ __align__(16) float smem[];
  pdl_trigger();
  pdl_wait();
  ChunkAt at;
  if (!sr_locate(p, &at)) return;
  const int head = blockIdx.x, dk = p.dk, dv = p.dv, tid = threadIdx.x;
  const int v0 = (dk + 3) & ~3, ldx = v0 + ((dv + 3) & ~3);      // columns of k, then of v
  __shared__ double c[SR_LONG];
  __shared__ float bt[SR_LONG], be[SR_LONG];
  float* lt = smem;                          // [SR_LONG columns j][SR_TP rows t]: L transposed
  float* X = lt + SR_LONG * SR_TP;           // [SR_LONG][ldx]
  float* kt = X + SR_LONG * ldx;             // [dk][SR_TP]
  if (tid < 32) {
    double sums[2];
    m.chunk_sums(p, head, at, sums);
    const double end = __shfl_sync(0xffffffffu, sums[1], 31);
    float* decays = m.decays + m.cell(p, at, head) * (SR_LONG + 4);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = tid + 32 * h;
      const float beta = t < at.count ? m.beta(p, head, at.first + t) : 0.f;
      c[t] = sums[h];
      bt[t] = beta;
      be[t] = beta * expf((float)sums[h]);
      decays[t] = t < at.count ? expf((float)(end - sums[h])) : 0.f;
    }
    if (tid == 0) decays[SR_LONG] = expf((float)end);
  }
  const Rows keys = m.keys(p, head, at), values{p.v + (size_t)at.first * p.v_ld + (size_t)head * dv, p.v_ld};
  sr_stage_transposed(kt, keys, dk, at.count);
  __syncthreads();
  // the right sides: rows of beta e^c k and beta v, zero past the last token and between the two
  const int warp = tid >> 5, lane = tid & 31;
  for (int t = warp; t < SR_LONG; t += DS_THREADS / 32) {
    const bool has = t < at.count;
    const float a = be[t], b = bt[t];
    float* x = X + t * ldx;
    for (int d = lane; d < v0; d += 32) x[d] = d < dk ? a * kt[d * SR_TP + t] : 0.f;
    for (int d = lane; d < ldx - v0; d += 32) x[v0 + d] = has && d < dv ? b * values.row(t)[d] : 0.f;
  }
  {
    const int row = 4 * (tid & 15), col = 4 * (tid >> 4);
    float a[4][4] = {};
    if (col <= row + 3) sr_mm44(a, kt, SR_TP, kt, SR_TP, dk, row, col);
#pragma unroll
    for (int b = 0; b < 4; ++b) {
      float l[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = row + e;
        l[e] = col + b < t ? a[e][b] * bt[t] * expf((float)(c[t] - c[col + b])) : 0.f;
      }
      store4(lt + (col + b) * SR_TP + row, l);
    }
  }
  const size_t cell = m.cell(p, at, head);
  for (int r0 = 0; r0 < SR_LONG; r0 += 16) {
    __syncthreads();
    if (r0 > 0) {
      const int row = r0 + 4 * (tid & 3);
      for (int col = 2 * (tid >> 2); col < ldx; col += DS_THREADS / 2) {
        float acc[4][2] = {};
#pragma unroll 8
        for (int j = 0; j < r0; ++j) {
          const float4 l = *reinterpret_cast<const float4*>(lt + j * SR_TP + row);
          const float2 x = *reinterpret_cast<const float2*>(X + j * ldx + col);
          acc[0][0] = fmaf(l.x, x.x, acc[0][0]), acc[0][1] = fmaf(l.x, x.y, acc[0][1]);
          acc[1][0] = fmaf(l.y, x.x, acc[1][0]), acc[1][1] = fmaf(l.y, x.y, acc[1][1]);
          acc[2][0] = fmaf(l.z, x.x, acc[2][0]), acc[2][1] = fmaf(l.z, x.y, acc[2][1]);
          acc[3][0] = fmaf(l.w, x.x, acc[3][0]), acc[3][1] = fmaf(l.w, x.y, acc[3][1]);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float2* x2 = reinterpret_cast<float2*>(X + (row + e) * ldx + col);
          *x2 = make_float2(x2->x - acc[e][0], x2->y - acc[e][1]);
        }
      }
      __syncthreads();
    }
    for (int i = tid; i < ldx; i += DS_THREADS) {
      float x[16];
#pragma unroll
      for (int t = 0; t < 16; ++t) x[t] = X[(r0 + t) * ldx + i];
#pragma unroll
      for (int j = 0; j < 15; ++j) {
        float l[16];
#pragma unroll
        for (int t = 0; t < 16; t += 4)
          if (t + 3 > j) load4(lt + (r0 + j) * SR_TP + r0 + t, l + t);
#pragma unroll
        for (int t = j + 1; t < 16; ++t) x[t] = fmaf(-l[t], x[j], x[t]);
      }
#pragma unroll
      for (int t = 0; t < 16; ++t) X[(r0 + t) * ldx + i] = x[t];
      if (i < dk) {
        float* dst = m.w + (cell * dk + i) * SR_LONG + r0;
#pragma unroll
        for (int t = 0; t < 16; t += 4) store4(dst + t, x + t);
      } else if (i >= v0 && i - v0 < dv) {
        float* dst = m.u + (cell * SR_LONG + r0) * dv + (i - v0);
#pragma unroll
        for (int t = 0; t < 16; ++t) dst[(size_t)t * dv] = x[t];
      }
    }
  }
}

// The chain over an entry's chunks for one head and COLS value columns: u = U - W S, then
// S <- e^(c_end) S + sum_j k_j (e^(c_end - c_j) u_j)^T.  The state's columns stay in shared memory;
// the next chunk's W and keys are on their way while a chunk is worked on.  Thread (rg, cg) of
// 16 x COLS / 2 owns four rows and two columns of a product; two such groups of threads take half of
// a product's depth each, the second one's share is added by (W S) or after (the state) the first's.
template <int COLS>
__device__ __forceinline__ void dc_mm42(float (&acc)[4][2], const float* xt, int ldx, const float* y, int depth, int row, int col) {
#pragma unroll 8
  for (int k = 0; k < depth; ++k) {
    const float4 x = *reinterpret_cast<const float4*>(xt + k * ldx + row);
    const float2 b = *reinterpret_cast<const float2*>(y + k * COLS + col);
    acc[0][0] = fmaf(x.x, b.x, acc[0][0]), acc[0][1] = fmaf(x.x, b.y, acc[0][1]);
    acc[1][0] = fmaf(x.y, b.x, acc[1][0]), acc[1][1] = fmaf(x.y, b.y, acc[1][1]);
    acc[2][0] = fmaf(x.z, b.x, acc[2][0]), acc[2][1] = fmaf(x.z, b.y, acc[2][1]);
    acc[3][0] = fmaf(x.w, b.x, acc[3][0]), acc[3][1] = fmaf(x.w, b.y, acc[3][1]);
  }
}

template <int COLS>
__global__ void __launch_bounds__(16 * COLS) delta_chain_kernel(const Delta m, const StateRun p, int* status) {
  extern __shared__ __align__(16) float smem[];
  pdl_trigger();
  pdl_wait();
  const int head = blockIdx.x, entry = blockIdx.y, col0 = blockIdx.z * COLS, tid = threadIdx.x;
  const int first = p.cu_tokens[entry], count = p.cu_tokens[entry + 1] - first;
  if (count < p.long_from) return;
  const int slot = p.slots[entry];
  if (slot < 0 || slot >= p.state_rows) {
    if (tid == 0 && blockIdx.z == 0) atomicOr(status, FE_STATUS_BAD_PAGE);
    return;
  }
  const int dk = p.dk, dv = p.dv, kp = (dk + 63) / 64 * 64;
  const int cols = min(COLS, dv - col0), half = dk * SR_LONG + SR_LONG * kp;
  float* S = smem;                           // [kp][COLS]
  float* us = S + kp * COLS;                 // [SR_LONG][COLS], weighted
  float* share = us + SR_LONG * COLS;        // [SR_LONG][COLS]: the second group's part of W S
  float* buffers = share + SR_LONG * COLS;   // 2 x (W transposed [dk][SR_LONG], keys [SR_LONG][kp])
  const int group = tid / (8 * COLS), mine = tid - group * 8 * COLS;
  const int row = 4 * (mine & 15), col = 2 * (mine >> 4);
  const int d_from = group == 0 ? 0 : dk / 2, d_count = group == 0 ? dk / 2 : dk - dk / 2;
  float* st = p.state + ((size_t)slot * p.heads + head) * dk * dv + col0;
  for (int i = tid; i < kp * COLS; i += blockDim.x) {
    const int d = i / COLS, c = i - d * COLS;
    S[i] = (d < dk && c < cols) ? st[(size_t)d * dv + c] : 0.f;
  }
  for (int i = tid; i < 2 * half; i += blockDim.x) buffers[i] = 0.f;      // key channels past dk stay zero
  __syncthreads();
  const int chunks = (count + SR_LONG - 1) / SR_LONG;
  const int lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
  const size_t cell0 = (size_t)sr_slot(first, entry, 0) * p.heads + head;
  const Rows keys{m.k_row(p, head, first), m.ld};
  const bool wide = keys.wide(dk);
  auto fetch = [&](int chunk, float* buf) {
    const float* w = m.w + (cell0 + (size_t)chunk * p.heads) * dk * SR_LONG;
    for (int i = 4 * tid; i < dk * SR_LONG; i += 4 * blockDim.x) sr_copy16(buf + i, w + i);
    const int have = min(SR_LONG, count - chunk * SR_LONG);
    float* ks = buf + dk * SR_LONG;
    for (int t = warp; t < SR_LONG; t += warps) {
      float* dst = ks + t * kp;
      if (t >= have) {
        for (int d = lane; d < dk; d += 32) dst[d] = 0.f;
      } else if (wide) {
        for (int d = 4 * lane; d < dk; d += 128) sr_copy16(dst + d, keys.row(chunk * SR_LONG + t) + d);
      } else {
        for (int d = lane; d < dk; d += 32) sr_copy4(dst + d, keys.row(chunk * SR_LONG + t) + d);
      }
    }
    sr_copy_commit();
  };
  fetch(0, buffers);
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const size_t cell = cell0 + (size_t)chunk * p.heads;
    const float* buf = buffers + (chunk & 1) * half;
    float* u = m.u + (cell * SR_LONG + row) * dv + col0 + col;
    const float* decays = m.decays + cell * (SR_LONG + 4);
    float x[4][2], w[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      w[e] = decays[row + e];
#pragma unroll
      for (int b = 0; b < 2; ++b) x[e][b] = group == 0 && col + b < cols ? u[(size_t)e * dv + b] : 0.f;
    }
    const float keep = decays[SR_LONG];
    sr_copy_wait<0>();
    __syncthreads();
    if (chunk + 1 < chunks) fetch(chunk + 1, buffers + ((chunk + 1) & 1) * half);
    float a[4][2] = {};
    dc_mm42<COLS>(a, buf + d_from * SR_LONG, SR_LONG, S + d_from * COLS, d_count, row, col);
    if (group == 1) {
#pragma unroll
      for (int e = 0; e < 4; ++e) *reinterpret_cast<float2*>(share + (row + e) * COLS + col) = make_float2(a[e][0], a[e][1]);
    }
    // the state before the chunk, for state_out
    float* dst = m.before + cell * dk * dv + col0;
    for (int i = tid; i < dk * COLS; i += blockDim.x) {
      const int d = i / COLS, c = i - d * COLS;
      if (c < cols) dst[(size_t)d * dv + c] = S[i];
    }
    __syncthreads();
    if (group == 0) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 more = *reinterpret_cast<const float2*>(share + (row + e) * COLS + col);
        x[e][0] -= a[e][0] + more.x;
        x[e][1] -= a[e][1] + more.y;
        *reinterpret_cast<float2*>(us + (row + e) * COLS + col) = make_float2(x[e][0] * w[e], x[e][1] * w[e]);
#pragma unroll
        for (int b = 0; b < 2; ++b)
          if (col + b < cols) u[(size_t)e * dv + b] = x[e][b];
      }
    }
    __syncthreads();
    const float* ks = buf + dk * SR_LONG;
    const int t_from = group * (SR_LONG / 2);
    for (int d0 = 0; d0 < kp; d0 += 64) {
      float b[4][2] = {};
      dc_mm42<COLS>(b, ks + t_from * kp + d0, kp, us + t_from * COLS, SR_LONG / 2, row, col);
      if (group == 0) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float2* s2 = reinterpret_cast<float2*>(S + (d0 + row + e) * COLS + col);
          const float2 old = *s2;
          *s2 = make_float2(fmaf(keep, old.x, b[e][0]), fmaf(keep, old.y, b[e][1]));
        }
      }
      __syncthreads();
      if (group == 1) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float2* s2 = reinterpret_cast<float2*>(S + (d0 + row + e) * COLS + col);
          const float2 old = *s2;
          *s2 = make_float2(old.x + b[e][0], old.y + b[e][1]);
        }
      }
    }
  }
  __syncthreads();
  for (int i = tid; i < dk * COLS; i += blockDim.x) {
    const int d = i / COLS, c = i - d * COLS;
    if (c < cols) st[(size_t)d * dv + c] = S[i];
  }
}

static size_t delta_solve_smem(int dk, int dv) {
  const size_t ldx = (size_t)((dk + 3) / 4 * 4) + (dv + 3) / 4 * 4;
  return sizeof(float) * ((size_t)SR_LONG * SR_TP + SR_LONG * ldx + (size_t)dk * SR_TP);
}
// Value columns of a block of delta_chain: few where the heads are small, so that there are more blocks.
static int delta_chain_cols(int dv) { return dv <= 64 ? 16 : 32; }
static size_t delta_chain_smem(int dk, int cols) {
  const size_t kp = (size_t)(dk + 63) / 64 * 64;
  return sizeof(float) * (kp * cols + (size_t)2 * SR_LONG * cols + 2 * ((size_t)dk * SR_LONG + SR_LONG * kp));
}
static bool delta_chunk_takes(int dk, int dv) {
  return chunk_takes(dk, dv, true) && delta_solve_smem(dk, dv) <= 200 * 1024 && delta_chain_smem(dk, delta_chain_cols(dv)) <= 200 * 1024;
}

FE_EXPORT long long fe_delta_rule_scratch(int tokens, int entries, int heads, int dk, int dv, int max_new) {
  const long long need = walk_in_stretches(dk, dv, 0) ? (long long)tokens * heads * dv : 0;
  if (max_new < SR_LONG_FROM || !delta_chunk_takes(dk, dv)) return need;
  return (need + 3) / 4 * 4 + sr_slots(tokens, entries) * heads * ((long long)dk * SR_LONG + (long long)SR_LONG * dv + (long long)dk * dv + SR_LONG + 4);
}

FE_EXPORT int fe_delta_rule(const float* qkv, long long ld, const float* gates, const float* gate, long long gate_ld,
                            const float* norm_w, float eps, float* state, int state_rows, const int* slots,
                            const int* cu_tokens, void* out, int out_dtype, int entries, int kv_heads, int heads, int dk, int dv,
                            int tokens, int max_new, float* scratch, int* status, cudaStream_t stream) {
  if (entries <= 0 || tokens <= 0) return 0;
  if (heads < 1 || kv_heads < 1 || heads % kv_heads || dk < 1 || dv < 1 || heads > 65535 || entries > 65535) return FE_ERR_BAD_SHAPE;
  StateRun p{state, state_rows, slots, cu_tokens, heads, dk, dv, 0, qkv + 2 * kv_heads * dk, ld, norm_w, 0, gate, gate_ld, 0, eps, out, nullptr, 0};
  Delta m{qkv, ld, kv_heads, heads / kv_heads, gates, nullptr, nullptr, nullptr, nullptr};
  if (walk_in_stretches(dk, dv, 0)) {
    p.raw = scratch;
    scratch = scratch ? scratch + ((size_t)tokens * heads * dv + 3) / 4 * 4 : nullptr;
  }
  const bool chunked = max_new >= SR_LONG_FROM && scratch != nullptr && delta_chunk_takes(dk, dv);
  if (chunked) p.long_from = SR_LONG_FROM;
  int rc = launch_walk(m, p, out_dtype, entries, tokens, status, stream);
  if (rc || !chunked) return rc ? rc : fe_last_error();
  const int chunks = (max_new + SR_LONG - 1) / SR_LONG;
  if (chunks > 65535) return FE_ERR_TOO_LARGE;
  const size_t cells = (size_t)sr_slots(tokens, entries) * heads;
  m.w = scratch;
  m.u = m.w + cells * dk * SR_LONG;
  m.decays = m.u + cells * SR_LONG * dv;
  m.before = m.decays + cells * (SR_LONG + 4);
  size_t smem = delta_solve_smem(dk, dv);
  cudaFuncSetAttribute(delta_solve_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  rc = fe_launch_dependent(delta_solve_kernel, dim3(heads, entries, chunks), dim3(DS_THREADS), smem, stream, m, p);
  if (rc) return rc;
  const int cols = delta_chain_cols(dv);
  smem = delta_chain_smem(dk, cols);
  const dim3 chain(heads, entries, (dv + cols - 1) / cols);
  if (cols == 16) {
    cudaFuncSetAttribute(delta_chain_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    rc = fe_launch_dependent(delta_chain_kernel<16>, chain, dim3(256), smem, stream, m, p, status);
  } else {
    cudaFuncSetAttribute(delta_chain_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    rc = fe_launch_dependent(delta_chain_kernel<32>, chain, dim3(512), smem, stream, m, p, status);
  }
  if (rc) return rc;
  rc = launch_out(m, p, out_dtype, entries, chunks, stream);
  return rc ? rc : fe_last_error();
}
