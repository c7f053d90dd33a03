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
  // i, f and the running sum F of f for a chunk's tokens lane and 32 + lane, by one warp; tokens
  // past the end have f = 0 and i = minus infinity
  struct Gates { double F[2]; float i[2]; };
  __device__ __forceinline__ Gates chunk_gates(const ChunkAt& at, int head) const {
    Gates g;
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = lane + 32 * h;
      float i = -INFINITY, f = 0.f;
      if (t < at.count) gates(at.first + t, head, &i, &f);
      g.i[h] = i, g.F[h] = (double)f;
    }
    sr_running_sum(g.F[0], g.F[1]);
    return g;
  }
  __device__ __forceinline__ const float* chunk(const StateRun& p, const ChunkAt& at, int head) const {
    return sums + ((size_t)at.slot * p.heads + head) * ((size_t)p.dk * p.dv + p.dk);
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
  __device__ __forceinline__ const float* start_norm(const StateRun& p, int head, const ChunkAt& at) const {
    return chunk(p, at, head) + (size_t)p.dk * p.dv;
  }
  // m_t = F_t + max(m before the chunk, the largest i_j - F_j up to t): the recurrence's maximum
  __device__ __forceinline__ void out_begin(const StateRun& p, int head, const ChunkAt& at, double* rt, double* ct, float* ea,
                                            float* fl) const {
    const int lane = threadIdx.x & 31;
    const size_t cell = (size_t)at.slot * p.heads + head;
    if (lane == 0 && at.first == at.entry_first)      // m after the entry's last token, now that nobody reads the one before its first
      top[(size_t)p.slots[blockIdx.y] * p.heads + head] = marks[cell * 4 + 3];
    const double m_start = (double)marks[cell * 4 + 2];
    const Gates g = chunk_gates(at, head);
    double big[2] = {(double)g.i[0] - g.F[0], (double)g.i[1] - g.F[1]};
    sr_running_max(big[0], big[1]);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = lane + 32 * h;
      const double F = g.F[h], m = F + fmax(m_start, big[h]);
      rt[t] = F - m;
      ct[t] = (double)g.i[h] - F;
      ea[t] = t < at.count ? expf((float)(F + m_start - m)) : 0.f;
      fl[t] = expf((float)-m);
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
  __shared__ float w[SR_LONG];
  float* ks = smem;                       // [SR_LONG][64]: 64 channels of the keys, weighted
  float* tile = ks + SR_LONG * 64;        // [SR_LONG][64]
  if (tid < 32) {
    const Memory::Gates g = m.chunk_gates(at, head);
    const double end = __shfl_sync(0xffffffffu, g.F[1], 31);
    float x[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) x[h] = (float)(end - g.F[h] + (double)g.i[h]);      // minus infinity past the end
    const float big = warp_max(fmaxf(x[0], x[1]));
#pragma unroll
    for (int h = 0; h < 2; ++h) w[tid + 32 * h] = expf((float)(end - g.F[h] + (double)g.i[h] - (double)big));
    if (tid == 0) {
      float* mark = m.marks + ((size_t)at.slot * p.heads + head) * 4;
      mark[0] = big;
      mark[1] = (float)end;
    }
  }
  float* sum = m.sums + ((size_t)at.slot * p.heads + head) * ((size_t)dk * dv + dk);
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
      if (c0 == 0 && tid < 64 && d0 + tid < dk) {
        float s = 0.f;
#pragma unroll 8
        for (int t = 0; t < SR_LONG; ++t) s += ks[t * 64 + tid];
        sum[(size_t)dk * dv + d0 + tid] = s;
      }
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

FE_EXPORT long long fe_matrix_memory_scratch(int tokens, int entries, int heads, int dk, int dv, int max_new) {
  const long long need = walk_in_stretches(dk, dv, 1) ? (long long)tokens * heads * dv : 0;
  if (max_new < SR_LONG_FROM || !chunk_takes(dk, dv, true)) return need;
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
  const bool chunked = max_new >= SR_LONG_FROM && scratch != nullptr && chunk_takes(dk, dv, true);
  if (chunked) p.long_from = SR_LONG_FROM;
  int rc = launch_walk(m, p, out_dtype, entries, tokens, status, stream);
  if (rc || !chunked) return rc ? rc : fe_last_error();
  const int chunks = (max_new + SR_LONG - 1) / SR_LONG;
  if (chunks > 65535) return FE_ERR_TOO_LARGE;
  m.sums = scratch;
  m.marks = m.sums + (size_t)sr_slots(tokens, entries) * heads * ((size_t)dk * dv + dk);
  const size_t smem = sizeof(float) * 2 * SR_LONG * 64;
  rc = fe_launch_dependent(memory_sums_kernel, dim3(heads, entries, chunks), dim3(256), smem, stream, m, p);
  if (rc) return rc;
  rc = fe_launch_dependent(memory_scan_kernel, dim3(heads, entries, (unsigned)(((long long)dk * dv + dk + 255) / 256)), dim3(256), 0, stream, m, p, status);
  if (rc) return rc;
  rc = launch_out(m, p, out_dtype, entries, chunks, stream);
  return rc ? rc : fe_last_error();
}
