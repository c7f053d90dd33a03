// A matrix memory with exponential gates and a normaliser, carried relative to a running maximum.
//
//     i = cap tanh((zi + bi) / cap),  f = logsigmoid(cap tanh((zf + bf) / cap))       per head
//     m_t = max(f + m_(t-1), i)                                            (m starts at zero)
//     S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T,   n_t likewise with k alone
//     o_t = S_t^T q / (max(|n_t . q|, e^(-m_t)) + 1e-6)
//
// then the head's norm, weight and gate.  q is the projection times dk^(-1/2).  In the walk the
// normaliser n is one more column of the state whose value is 1 for every token.  Chunk form, with
// F_t the sum of f from the chunk's first token up to t and S, n, m those before the chunk:
//     S_t e^(m_t) = e^(F_t + m) S + sum_(j <= t) e^(F_t - F_j + i_j) k_j v_j^T
// memory_sums takes the second term at the chunk's end, relative to its own maximum; memory_scan
// chains S, n and m over the chunks; state_out takes the outputs (m_t by its own recurrence).
#include "state_recurrence.cuh"

struct Memory {
  const float *q, *k;       // projections, token t at t * ld + head * dk
  long long ld;
  const float *zi, *zf;     // token t, head h at t * gates_ld + h
  long long gates_ld;
  const float *bi, *bf;     // [heads]
  float cap, q_scale;
  float* norm;              // [rows, heads, dk]
  float* top;               // [rows, heads]
  // chunk-parallel scratch
  float* sums;              // [slots, heads, dk * dv + dk]: what a chunk adds to S and n, then (scan) S and n before it
  float* marks;             // [slots, heads, 4]: the sums' own maximum, F at the chunk's end, then m before the chunk

  static constexpr int VECS = 2, SCALARS = 3, EXTRA = 1;
  static constexpr bool SCORES = true, NORMALISER = true;

  __device__ __forceinline__ void gates(int token, int head, float* i, float* f) const {
    *i = cap * tanhf((zi[(size_t)token * gates_ld + head] + bi[head]) / cap);
    *f = -sr_softplus(-cap * tanhf((zf[(size_t)token * gates_ld + head] + bf[head]) / cap));
  }
  __device__ __forceinline__ float* column(const StateRun& p, int slot, int head, int col, size_t* step) const {
    const size_t cell = (size_t)slot * p.heads + head;
    if (col == p.dv) {
      *step = 1;
      return norm + cell * p.dk;
    }
    *step = p.dv;
    return p.state + cell * p.dk * p.dv + col;
  }
  __device__ __forceinline__ void begin(const StateRun& p, int slot, int head, float* carry) const {
    if (threadIdx.x == 0) carry[0] = top[(size_t)slot * p.heads + head];
  }
  __device__ __forceinline__ void end(const StateRun& p, int slot, int head, const float* carry) const {
    if (threadIdx.x == 0) top[(size_t)slot * p.heads + head] = carry[0];
  }
  __device__ __forceinline__ void stage(const StateRun& p, int head, int first, int nt, float* vec, int pitch, float* sc) const {
    for (int i = threadIdx.x; i < nt * p.dk; i += blockDim.x) {
      const int t = i / p.dk, d = i - t * p.dk;
      const size_t at = (size_t)(first + t) * ld + (size_t)head * p.dk + d;
      float* dst = vec + t * VECS * pitch + d;
      dst[0] = q[at] * q_scale, dst[pitch] = k[at];
    }
    if (threadIdx.x < 32) {
      const int lane = threadIdx.x;
      float li = 0.f, lf = 0.f;
      if (lane < nt) gates(first + lane, head, &li, &lf);
      float* carry = sc + SR_CHUNK * SCALARS;
      float m = carry[0];
      for (int t = 0; t < nt; ++t) {
        const float i = __shfl_sync(0xffffffffu, li, t), f = __shfl_sync(0xffffffffu, lf, t);
        const float next = fmaxf(f + m, i);
        if (lane == 0) {
          sc[t * SCALARS + 0] = expf(f + m - next);
          sc[t * SCALARS + 1] = expf(i - next);
          sc[t * SCALARS + 2] = expf(-next);
        }
        m = next;
      }
      __syncwarp();
      if (lane == 0) carry[0] = m;
    }
  }
  template <int KPT>
  __device__ __forceinline__ float step(float (&S)[KPT], const float* vec, int pitch, const float* sc, float value, int s, int ds) const {
    const float *qs = vec + s, *ks = qs + pitch;
    const float keep = sc[0], write = sc[1] * value;
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
      S[i] = fmaf(keep, S[i], ks[i * ds] * write);
      acc = fmaf(S[i], qs[i * ds], acc);
    }
    return sr_column_sum(acc, ds);
  }
  __device__ __forceinline__ float scale(const float* o, const float* sc, int dv) const {
    return 1.f / (fmaxf(fabsf(o[dv]), sc[2]) + 1e-6f);
  }

  // -- chunk form --
  // F (sums of f up to every token) and i of a chunk in shared memory, by one warp; tokens past
  // the end keep F and have i = 0
  __device__ __forceinline__ void chunk_gates(const ChunkAt& at, int head, double* F, float* i_log, float* f_log) const {
    const int tid = threadIdx.x;
    if (tid < SR_LONG) {
      float i = 0.f, f = 0.f;
      if (tid < at.count) gates(at.first + tid, head, &i, &f);
      i_log[tid] = i, f_log[tid] = f;
    }
    __syncthreads();
    if (tid == 0) {
      double sum = 0.0;
      for (int t = 0; t < SR_LONG; ++t) {
        sum += (double)f_log[t];
        F[t] = sum;
      }
    }
    __syncthreads();
  }
  __device__ __forceinline__ const float* chunk(const StateRun& p, const ChunkAt& at, int head) const {
    return sums + ((size_t)at.slot * p.heads + head) * ((size_t)p.dk * p.dv + p.dk);
  }
  __device__ __forceinline__ float query(const StateRun& p, int head, const ChunkAt& at, int t, int d) const {
    return q[(size_t)(at.first + t) * ld + (size_t)head * p.dk + d] * q_scale;
  }
  __device__ __forceinline__ float key(const StateRun& p, int head, const ChunkAt& at, int t, int d) const {
    return k[(size_t)(at.first + t) * ld + (size_t)head * p.dk + d];
  }
  __device__ __forceinline__ float other(const StateRun& p, int head, const ChunkAt& at, int t, int c) const {
    return p.v[(size_t)(at.first + t) * p.v_ld + (size_t)head * p.dv + c];
  }
  __device__ __forceinline__ float start(const StateRun& p, int head, const ChunkAt& at, int d, int c) const {
    return chunk(p, at, head)[(size_t)d * p.dv + c];
  }
  __device__ __forceinline__ float start_norm(const StateRun& p, int head, const ChunkAt& at, int d) const {
    return chunk(p, at, head)[(size_t)p.dk * p.dv + d];
  }
  __device__ __forceinline__ void out_begin(const StateRun& p, int head, const ChunkAt& at, double* rt, double* ct, float* ea,
                                            float* fl) const {
    __shared__ float i_log[SR_LONG], f_log[SR_LONG];
    chunk_gates(at, head, rt, i_log, f_log);          // rt holds F for now
    if (threadIdx.x == 0) {
      if (at.first == at.entry_first)      // m after the entry's last token, now that nobody reads the one before its first
        top[(size_t)p.slots[blockIdx.y] * p.heads + head] = marks[((size_t)at.slot * p.heads + head) * 4 + 3];
      const float m_start = marks[((size_t)at.slot * p.heads + head) * 4 + 2];
      float m = m_start;
      for (int t = 0; t < SR_LONG; ++t) {
        m = fmaxf(f_log[t] + m, i_log[t]);
        const double F = rt[t];
        ct[t] = (double)i_log[t] - F;
        ea[t] = t < at.count ? expf((float)(F + (double)m_start - (double)m)) : 0.f;
        fl[t] = expf(-m);
        rt[t] = F - (double)m;
      }
    }
  }
};

// What a chunk adds to S and n by its end, relative to the sums' own maximum.
__global__ void __launch_bounds__(256) memory_sums_kernel(const Memory m, const StateRun p) {
  extern __shared__ __align__(16) float smem[];
  pdl_trigger();
  pdl_wait();
  ChunkAt at;
  if (!sr_locate(p, &at)) return;
  const int head = blockIdx.x, dk = p.dk, dv = p.dv, tid = threadIdx.x;
  __shared__ double F[SR_LONG];
  __shared__ float i_log[SR_LONG], f_log[SR_LONG], w[SR_LONG];
  const int kp = (dk + 63) / 64 * 64;
  float* ks = smem;                       // [SR_LONG][kp], weighted
  float* tile = ks + SR_LONG * kp;        // [SR_LONG][64]
  m.chunk_gates(at, head, F, i_log, f_log);
  if (tid < 32) {
    const double end = F[at.count - 1];
    float big = -INFINITY;
    for (int t = tid; t < at.count; t += 32) big = fmaxf(big, (float)(end - F[t] + (double)i_log[t]));
    big = warp_max(big);
    for (int t = tid; t < SR_LONG; t += 32)
      w[t] = t < at.count ? expf((float)(end - F[t] + (double)i_log[t] - (double)big)) : 0.f;
    if (tid == 0) {
      float* mark = m.marks + ((size_t)at.slot * p.heads + head) * 4;
      mark[0] = big;
      mark[1] = (float)end;
    }
  }
  __syncthreads();
  for (int i = tid; i < SR_LONG * kp; i += blockDim.x) {
    const int t = i / kp, d = i - t * kp;
    ks[i] = (t < at.count && d < dk) ? m.key(p, head, at, t, d) * w[t] : 0.f;
  }
  __syncthreads();
  float* sum = m.sums + ((size_t)at.slot * p.heads + head) * ((size_t)dk * dv + dk);
  for (int d = tid; d < dk; d += blockDim.x) {
    float s = 0.f;
    for (int t = 0; t < at.count; ++t) s += ks[t * kp + d];
    sum[(size_t)dk * dv + d] = s;
  }
  const int row = 4 * (tid & 15), col = 4 * (tid >> 4);
  for (int c0 = 0; c0 < dv; c0 += 64) {
    __syncthreads();
    for (int i = tid; i < SR_LONG * 64; i += blockDim.x) {
      const int t = i >> 6, c = c0 + (i & 63);
      tile[i] = (t < at.count && c < dv) ? m.other(p, head, at, t, c) : 0.f;
    }
    __syncthreads();
    for (int d0 = 0; d0 < dk; d0 += 64) {
      float acc[4][4] = {};
      sr_mm44(acc, ks + d0, kp, tile, 64, at.count, row, col);
#pragma unroll
      for (int a = 0; a < 4; ++a) {
        const int d = d0 + row + a;
        if (d >= dk) continue;
#pragma unroll
        for (int b = 0; b < 4; ++b)
          if (c0 + col + b < dv) sum[(size_t)d * dv + c0 + col + b] = acc[a][b];
      }
    }
  }
}

// One thread per element of (S, n) walks an entry's chunks.
__global__ void __launch_bounds__(256) memory_scan_kernel(const Memory m, const StateRun p, int* status) {
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
  const size_t cells = (size_t)p.dk * p.dv, size = cells + p.dk;
  const size_t cell = (size_t)blockIdx.z * blockDim.x + threadIdx.x;
  if (cell >= size) return;
  const int chunks = (count + SR_LONG - 1) / SR_LONG;
  const size_t mine = (size_t)slot * p.heads + head, base = (size_t)sr_slot(first, entry, 0) * p.heads + head;
  float* st = cell < cells ? p.state + mine * cells + cell : m.norm + mine * p.dk + (cell - cells);
  float* sum = m.sums + base * size + cell;
  float* marks = m.marks + base * 4;
  const size_t stride = (size_t)p.heads * size;
  float state = *st, top = m.top[mine];
  for (int c0 = 0; c0 < chunks; c0 += 8) {
    float add[8], big[8], fall[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const bool has = c0 + j < chunks;
      add[j] = has ? sum[(size_t)(c0 + j) * stride] : 0.f;
      big[j] = has ? marks[(size_t)(c0 + j) * p.heads * 4] : 0.f;
      fall[j] = has ? marks[(size_t)(c0 + j) * p.heads * 4 + 1] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c0 + j < chunks) {
        sum[(size_t)(c0 + j) * stride] = state;
        if (cell == 0) marks[(size_t)(c0 + j) * p.heads * 4 + 2] = top;
        const float next = fmaxf(fall[j] + top, big[j]);
        state = fmaf(expf(fall[j] + top - next), state, expf(big[j] - next) * add[j]);
        top = next;
      }
    }
  }
  *st = state;
  // m of the request is read by every block here: the next launch stores it (out_begin of chunk 0)
  if (cell == 0) marks[3] = top;
}

static size_t memory_sums_smem(int dk) { return sizeof(float) * (size_t)SR_LONG * ((dk + 63) / 64 * 64 + 64); }

FE_EXPORT long long fe_matrix_memory_scratch(int tokens, int entries, int heads, int dk, int dv, int max_new) {
  const long long need = walk_in_stretches(dk, dv, 1) ? (long long)tokens * heads * dv : 0;
  if (max_new < SR_LONG_FROM || !chunk_takes(dk, dv, true) || memory_sums_smem(dk) > 200 * 1024) return need;
  return need + sr_slots(tokens, entries) * heads * ((long long)dk * dv + dk + 4);
}

FE_EXPORT int fe_matrix_memory(const float* proj, long long ld, int q_off, int k_off, int v_off, int g_off, int i_off,
                               int f_off, const float* bi, const float* bf, float cap, float q_scale, const float* norm_w,
                               float eps, float* state, float* norm, float* top, int state_rows, const int* slots,
                               const int* cu_tokens, void* out, int out_dtype, int entries, int heads, int dk, int dv,
                               int tokens, int max_new, float* scratch, int* status, cudaStream_t stream) {
  if (entries <= 0 || tokens <= 0) return 0;
  if (heads < 1 || dk < 1 || dv < 1 || heads > 65535 || entries > 65535 || !(cap > 0.f)) return FE_ERR_BAD_SHAPE;
  StateRun p{state, state_rows, slots, cu_tokens, heads, dk, dv, 0, proj + v_off, ld, norm_w, dv, proj + g_off, ld, 1, eps, out, nullptr, 0};
  Memory m{proj + q_off, proj + k_off, ld, proj + i_off, proj + f_off, ld, bi, bf, cap, q_scale, norm, top, nullptr, nullptr};
  if (walk_in_stretches(dk, dv, 1)) {
    p.raw = scratch;
    scratch = scratch ? scratch + (size_t)tokens * heads * dv : nullptr;
  }
  const bool chunked = max_new >= SR_LONG_FROM && scratch != nullptr && chunk_takes(dk, dv, true) && memory_sums_smem(dk) <= 200 * 1024;
  if (chunked) p.long_from = SR_LONG_FROM;
  int rc = launch_walk(m, p, out_dtype, entries, tokens, status, stream);
  if (rc || !chunked) return rc ? rc : fe_last_error();
  const int chunks = (max_new + SR_LONG - 1) / SR_LONG;
  if (chunks > 65535) return FE_ERR_TOO_LARGE;
  m.sums = scratch;
  m.marks = m.sums + (size_t)sr_slots(tokens, entries) * heads * ((size_t)dk * dv + dk);
  const size_t smem = memory_sums_smem(dk);
  cudaFuncSetAttribute(memory_sums_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  rc = fe_launch_dependent(memory_sums_kernel, dim3(heads, entries, chunks), dim3(256), smem, stream, m, p);
  if (rc) return rc;
  rc = fe_launch_dependent(memory_scan_kernel, dim3(heads, entries, (unsigned)(((long long)dk * dv + dk + 255) / 256)), dim3(256), 0, stream, m, p, status);
  if (rc) return rc;
  rc = launch_out(m, p, out_dtype, entries, chunks, stream);
  return rc ? rc : fe_last_error();
}
