// Retention: linear attention with a fixed decay per head, queries and keys rotated by position.
//
//     S_t = d S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t          per head, d in [0, 1]
//
// then the head's root mean square, an optional weight and the gate silu(.).  A factor of the keys is
// carried by the queries (`q_scale`), which read the state.  The walk rotates q and k itself as it
// stages them (`table`); for steps with long portions they come rotated.  Chunk form, with S the
// state before a chunk of n tokens and t, j counting inside it from zero:
//     o_t = d^(t + 1) S^T q_t + sum_(j <= t) d^(t - j) (k_j . q_t) v_j
//     S'  = d^n S + sum_j d^(n - 1 - j) k_j v_j^T
// retention_sums takes the last sum for all chunks side by side, retention_scan chains the states,
// state_out takes the outputs.
#include "state_recurrence.cuh"

struct Retention {
  const float *q, *k;       // projections, token t at t * ld + head * dk
  long long ld;
  float q_scale;
  const float* decay;       // [heads]
  const float2* table;      // or null: cosine and sine, [tokens, rot / 2]
  int rot, interleaved;     // leading elements of a head that are rotated
  float* sums;              // chunk form: [slots, heads, dk * dv], what a chunk adds, then (scan) the state before it

  static constexpr int VECS = 2, SCALARS = 1, EXTRA = 0;
  static constexpr bool SCORES = true, NORMALISER = false;

  __device__ __forceinline__ float* column(const StateRun& p, int slot, int head, int col, size_t* step) const {
    *step = p.dv;
    return p.state + ((size_t)slot * p.heads + head) * p.dk * p.dv + col;
  }
  __device__ __forceinline__ void begin(const StateRun&, int, int, float*) const {}
  __device__ __forceinline__ void end(const StateRun&, int, int, const float*) const {}
  __device__ __forceinline__ void stage(const StateRun& p, int head, int first, int nt, float* vec, int pitch, float* sc) const {
    const int half = rot >> 1;
    for (int i = threadIdx.x; i < nt * p.dk; i += blockDim.x) {
      const int t = i / p.dk, d = i - t * p.dk;
      const size_t row = (size_t)(first + t) * ld + (size_t)head * p.dk;
      float qd = q[row + d], kd = k[row + d];
      if (table != nullptr && d < rot) {
        // element d of the rotated pair: a cos - b sin for the first of the two, a cos + b sin for the second
        const bool second = interleaved ? (d & 1) != 0 : d >= half;
        const int pair = interleaved ? d >> 1 : second ? d - half : d;
        const int other = interleaved ? d ^ 1 : second ? d - half : d + half;
        const float2 cs = table[(size_t)(first + t) * half + pair];
        const float s = second ? cs.y : -cs.y;
        qd = qd * cs.x + q[row + other] * s;
        kd = kd * cs.x + k[row + other] * s;
      }
      float* dst = vec + t * VECS * pitch + d;
      dst[0] = qd * q_scale, dst[pitch] = kd;
    }
    for (int t = threadIdx.x; t < nt; t += blockDim.x) sc[t] = decay[head];
  }
  template <int KPT>
  __device__ __forceinline__ float step(float (&S)[KPT], const float* vec, int pitch, const float* sc, float value, int s, int ds) const {
    const float *qs = vec + s, *ks = qs + pitch;
    const float keep = sc[0];
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
      S[i] = fmaf(keep, S[i], ks[i * ds] * value);
      acc = fmaf(S[i], qs[i * ds], acc);
    }
    return sr_column_sum(acc, ds);
  }
  __device__ __forceinline__ float scale(const float*, const float*, int) const { return 1.f; }

  // -- chunk form --
  // The logarithm of the decay, kept finite: sums of it are subtracted from one another, and any
  // positive power of a decay of zero is zero all the same.
  __device__ __forceinline__ double log_decay(int head) const { return fmax(log((double)decay[head]), -1e4); }
  __device__ __forceinline__ const float* chunk(const StateRun& p, const ChunkAt& at, int head) const {
    return sums + ((size_t)at.slot * p.heads + head) * (size_t)p.dk * p.dv;
  }
  __device__ __forceinline__ Rows queries(const StateRun& p, int head, const ChunkAt& at) const {
    return Rows{q + (size_t)at.first * ld + (size_t)head * p.dk, ld};
  }
  __device__ __forceinline__ float query_mul() const { return q_scale; }
  __device__ __forceinline__ Rows keys(const StateRun& p, int head, const ChunkAt& at) const {
    return Rows{k + (size_t)at.first * ld + (size_t)head * p.dk, ld};
  }
  __device__ __forceinline__ Rows others(const StateRun& p, int head, const ChunkAt& at) const {
    return Rows{p.v + (size_t)at.first * p.v_ld + (size_t)head * p.dv, p.v_ld};
  }
  __device__ __forceinline__ Rows starts(const StateRun& p, int head, const ChunkAt& at) const { return Rows{chunk(p, at, head), p.dv}; }
  __device__ __forceinline__ void out_begin(const StateRun& p, int head, const ChunkAt& at, double* rt, double* ct, float* ea, float*) const {
    const double l = log_decay(head);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = (threadIdx.x & 31) + 32 * h;
      rt[t] = l * t;
      ct[t] = -l * t;
      ea[t] = t < at.count ? expf((float)(l * (t + 1))) : 0.f;
    }
  }
};

// What a chunk adds to the state by its end.
__global__ void __launch_bounds__(256) retention_sums_kernel(const Retention m, const StateRun p) {
  extern __shared__ __align__(16) float smem[];
  pdl_trigger();
  pdl_wait();
  ChunkAt at;
  if (!sr_locate(p, &at)) return;
  const int head = blockIdx.x, dk = p.dk, dv = p.dv, tid = threadIdx.x;
  __shared__ float w[SR_LONG];
  float* ks = smem;                       // [SR_LONG][64]: 64 channels of the keys, weighted
  float* tile = ks + SR_LONG * 64;        // [SR_LONG][64]
  if (tid < SR_LONG) w[tid] = tid < at.count ? expf((float)(m.log_decay(head) * (at.count - 1 - tid))) : 0.f;
  float* sum = m.sums + ((size_t)at.slot * p.heads + head) * (size_t)dk * dv;
  const bool wide = (dv & 3) == 0 && ((uintptr_t)sum & 15) == 0;
  const int row = 4 * (tid & 15), col = 4 * (tid >> 4);
  const Rows keys = m.keys(p, head, at), values = m.others(p, head, at);
  for (int d0 = 0; d0 < dk; d0 += 64) {
    __syncthreads();
    sr_stage_columns(ks, keys, SR_LONG, at.count, d0, dk);
    __syncthreads();
    for (int i = tid; i < SR_LONG * 64; i += blockDim.x) ks[i] *= w[i >> 6];
    for (int c0 = 0; c0 < dv; c0 += 64) {
      __syncthreads();
      sr_stage_columns(tile, values, SR_LONG, at.count, c0, dv);
      __syncthreads();
      float acc[4][4] = {};
      sr_mm44(acc, ks, 64, tile, 64, at.count, row, col);
#pragma unroll
      for (int a = 0; a < 4; ++a) {
        const int d = d0 + row + a;
        if (d >= dk) continue;
        float* dst = sum + (size_t)d * dv + c0 + col;
        if (wide && c0 + col < dv) {
          store4(dst, acc[a]);
        } else if (!wide) {
#pragma unroll
          for (int b = 0; b < 4; ++b)
            if (c0 + col + b < dv) dst[b] = acc[a][b];
        }
      }
    }
  }
}

// One thread per element of S walks an entry's chunks.
__global__ void __launch_bounds__(256) retention_scan_kernel(const Retention m, const StateRun p, int* status) {
  pdl_trigger();
  pdl_wait();
  const int head = blockIdx.x, entry = blockIdx.y;
  const int first = p.cu_tokens[entry], count = p.cu_tokens[entry + 1] - first;
  if (count < p.long_from) return;
  const int slot = p.slots[entry];
  if (slot < 0 || slot >= p.state_rows) {
    if (threadIdx.x == 0 && blockIdx.z == 0) atomicOr(status, FE_STATUS_BAD_PAGE);
    return;
  }
  const size_t size = (size_t)p.dk * p.dv, cell = (size_t)blockIdx.z * blockDim.x + threadIdx.x;
  if (cell >= size) return;
  const int chunks = (count + SR_LONG - 1) / SR_LONG;
  float* st = p.state + ((size_t)slot * p.heads + head) * size + cell;
  float* sum = m.sums + ((size_t)sr_slot(first, entry, 0) * p.heads + head) * size + cell;
  const size_t stride = (size_t)p.heads * size;
  const double l = m.log_decay(head);
  const float whole = expf((float)(l * SR_LONG)), rest = expf((float)(l * (count - (chunks - 1) * SR_LONG)));
  float state = *st;
  for (int c0 = 0; c0 < chunks; c0 += 8) {               // eight chunks' sums are fetched before any is replaced
    float add[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) add[j] = c0 + j < chunks ? sum[(size_t)(c0 + j) * stride] : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c0 + j < chunks) {
        sum[(size_t)(c0 + j) * stride] = state;
        state = fmaf(c0 + j + 1 < chunks ? whole : rest, state, add[j]);
      }
    }
  }
  *st = state;
}

FE_EXPORT long long fe_retention_scratch(int tokens, int entries, int heads, int dk, int dv, int max_new) {
  const long long need = walk_in_stretches(dk, dv, 0) ? ((long long)tokens * heads * dv + 3) / 4 * 4 : 0;
  if (max_new < SR_LONG_FROM || !chunk_takes(dk, dv, true)) return need;
  return need + sr_slots(tokens, entries) * heads * (long long)dk * dv;
}

// `table` (or null) rotates the leading `rot` elements of every q and k head in the walk only: entries of
// SR_LONG_FROM tokens or more need q and k rotated beforehand (and no table).
FE_EXPORT int fe_retention(const float* proj, long long ld, int q_off, int k_off, int v_off, int g_off, float q_scale,
                           const float* decay, const float* table, int rot, int interleaved, const float* norm_w, float eps,
                           float* state, int state_rows, const int* slots, const int* cu_tokens, void* out, int out_dtype,
                           int entries, int heads, int dk, int dv, int tokens, int max_new, float* scratch, int* status,
                           cudaStream_t stream) {
  if (entries <= 0 || tokens <= 0) return 0;
  if (heads < 1 || dk < 1 || dv < 1 || heads > 65535 || entries > 65535) return FE_ERR_BAD_SHAPE;
  if (table != nullptr && (rot < 2 || rot % 2 || rot > dk || max_new >= SR_LONG_FROM)) return FE_ERR_BAD_SHAPE;
  StateRun p{state, state_rows, slots, cu_tokens, heads, dk, dv, 0, proj + v_off, ld, norm_w, 0, proj + g_off, ld, 0, eps, out, nullptr, 0};
  Retention m{proj + q_off, proj + k_off, ld, q_scale, decay, (const float2*)table, rot, interleaved, nullptr};
  if (walk_in_stretches(dk, dv, 0)) {
    p.raw = scratch;
    scratch = scratch ? scratch + ((size_t)tokens * heads * dv + 3) / 4 * 4 : nullptr;
  }
  const bool chunked = max_new >= SR_LONG_FROM && scratch != nullptr && chunk_takes(dk, dv, true);
  if (chunked) p.long_from = SR_LONG_FROM;
  int rc = launch_walk(m, p, out_dtype, entries, tokens, status, stream);
  if (rc || !chunked) return rc ? rc : fe_last_error();
  const int chunks = (max_new + SR_LONG - 1) / SR_LONG;
  if (chunks > 65535) return FE_ERR_TOO_LARGE;
  m.sums = scratch;
  rc = fe_launch_dependent(retention_sums_kernel, dim3(heads, entries, chunks), dim3(256), sizeof(float) * 2 * SR_LONG * 64, stream, m, p);
  if (rc) return rc;
  rc = fe_launch_dependent(retention_scan_kernel, dim3(heads, entries, (unsigned)(((long long)dk * dv + 255) / 256)), dim3(256), 0, stream, m, p, status);
  if (rc) return rc;
  rc = launch_out(m, p, out_dtype, entries, chunks, stream);
  return rc ? rc : fe_last_error();
}
