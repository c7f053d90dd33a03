// Time mixing with a state per head whose decay depends on the token, per key channel ("wkv").
//
//     o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t,      S_t = diag(w_t) S_(t-1) + k_t v_t^T
//     w_t = exp(-exp(b + A tanh(z_t))),  z_t a low-rank projection of the token
//
// Every projection reads a mix h + (h' - h) mu of the token's normalised row h and the one before
// it, h'.  A head's o is divided by its root mean square, weighted and gated.
//
//   token_shift      the mixes of all projections and the row itself, rounded once, from 32-bit
//                    rows; the last row of an entry is left in the request's state.  For steps in
//                    which every entry brings one token the residual sum and the norm are taken in
//                    the same launch.
//   wkv_decay        w_t for all tokens and channels.
//   state_walk       (state_recurrence.cuh) short entries.
//   wkv_local / wkv_scan / state_out   long entries, chunk by chunk side by side: with b_t the product of
//                    the decays from the chunk's first token up to t,
//                      S_t = diag(b_t) S_start + S_local_t,   o_t = (r_t b_(t-1))^T S_start + o_local_t.
//                    No division by a decay anywhere (it may be as small as exp(-exp(.)) gets).
#include "state_recurrence.cuh"

// ---------------------------------------------------------------------------
// token_shift
// ---------------------------------------------------------------------------
// y: the normalised rows, 32-bit [tokens, width], or null: then row t is residual + update + shift
// (written back), normalised here, and every entry brings one token.
// V: neighbouring elements a thread takes at a time.
template <int V> __device__ __forceinline__ void ts_load(const float* p, float* v) { if constexpr (V == 4) load4(p, v); else v[0] = p[0]; }
template <int V> __device__ __forceinline__ void ts_load(const bf16* p, float* v) { if constexpr (V == 4) load4(p, v); else v[0] = to_float(p[0]); }
template <int V> __device__ __forceinline__ void ts_store(float* p, const float* v) { if constexpr (V == 4) store4(p, v); else p[0] = v[0]; }
template <int V> __device__ __forceinline__ void ts_store(bf16* p, const float* v) { if constexpr (V == 4) store4(p, v); else p[0] = from_float<bf16>(v[0]); }

template <typename TU, typename TO, int V>
__global__ void __launch_bounds__(1024)
token_shift_kernel(const float* __restrict__ y, float* __restrict__ residual, const TU* __restrict__ update,
                   const float* __restrict__ shift, long long shift_stride, const float* __restrict__ weight, float eps,
                   const float* __restrict__ mu, int mixes, float* __restrict__ state, const int* __restrict__ slots,
                   const int* __restrict__ cu_tokens, const int* __restrict__ token_entry, TO* __restrict__ mixed,
                   TO* __restrict__ plain, int n_tokens, int width) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int entry = token_entry[t];
  const int first = cu_tokens[entry], last = cu_tokens[entry + 1] - 1;
  float* st = state + (size_t)slots[entry] * width;
  const float* mine = row;
  float inv = 1.f;
  if (y == nullptr) {
    float* res = residual + (size_t)t * width;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
      float x[V], u[V];
      ts_load<V>(res + i, x);
      if (update != nullptr) {
        ts_load<V>(update + (size_t)t * width + i, u);
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] += u[e];
      }
      if (shift != nullptr) {
        ts_load<V>(shift + (size_t)t * shift_stride + i, u);
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] += u[e];
      }
      ts_store<V>(res + i, x);
      ts_store<V>(row + i, x);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(x[e], x[e], ss);
    }
    inv = rsqrtf(block_sum(ss, scratch) / (float)width + eps);
  } else {
    mine = y + (size_t)t * width;
  }
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    float h[V], d[V], w[V];
    ts_load<V>(mine + i, h);
    // only the block of an entry's first token touches the state: it reads it, then leaves the last row
    ts_load<V>(t == first ? st + i : y + (size_t)(t - 1) * width + i, d);
    if (y == nullptr) {
      ts_load<V>(weight + i, w);
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] = h[e] * inv * w[e];
    }
    if (t == first) {
      if (t != last) ts_load<V>(y + (size_t)last * width + i, w);
      ts_store<V>(st + i, t == last ? h : w);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) d[e] -= h[e];
#pragma unroll 5
    for (int j = 0; j < mixes; ++j) {
      float m[V];
      ts_load<V>(mu + (size_t)j * width + i, m);
#pragma unroll
      for (int e = 0; e < V; ++e) m[e] = fmaf(d[e], m[e], h[e]);
      ts_store<V>(mixed + ((size_t)j * n_tokens + t) * width + i, m);
    }
    if (plain != nullptr) ts_store<V>(plain + (size_t)t * width + i, h);
  }
}

FE_EXPORT int fe_token_shift(const float* y, float* residual, const void* update, int update_dtype, const float* shift,
                             long long shift_stride, const float* weight, float eps, const float* mu, int mixes,
                             float* state, const int* slots, const int* cu_tokens, const int* token_entry, void* mixed,
                             void* plain, int out_dtype, int n_tokens, int width, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (width < 1 || mixes < 1 || (y == nullptr && (residual == nullptr || weight == nullptr))) return FE_ERR_BAD_SHAPE;
  const size_t smem = y == nullptr ? (size_t)width * sizeof(float) : 0;
  if (smem > 200 * 1024) return FE_ERR_TOO_LARGE;
  int rc = FE_ERR_BAD_DTYPE;
  if (update == nullptr) update_dtype = FE_DTYPE_F32;
  const bool wide = width % 4 == 0 && shift_stride % 4 == 0 &&
                    (((uintptr_t)y | (uintptr_t)residual | (uintptr_t)update | (uintptr_t)shift | (uintptr_t)weight | (uintptr_t)mu |
                      (uintptr_t)state | (uintptr_t)mixed | (uintptr_t)plain) & 15) == 0;
  const int items = wide ? width / 4 : width;
  const int threads = items >= 1024 ? 1024 : (items + 31) / 32 * 32;
#define SHIFT_V(TU, TO, V)                                                                                             \
  do {                                                                                                                 \
    if (smem > 47 * 1024)                                                                                              \
      cudaFuncSetAttribute(token_shift_kernel<TU, TO, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
    rc = fe_launch_dependent(token_shift_kernel<TU, TO, V>, dim3(n_tokens), dim3(threads), smem, stream, y, residual,  \
                             (const TU*)update, shift, shift_stride, weight, eps, mu, mixes, state, slots, cu_tokens,  \
                             token_entry, (TO*)mixed, (TO*)plain, n_tokens, width);                                    \
  } while (0)
#define SHIFT(TU, TO)                \
  do {                               \
    if (wide) SHIFT_V(TU, TO, 4);    \
    else SHIFT_V(TU, TO, 1);         \
  } while (0)
  if (update_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_F32) SHIFT(float, float);
  else if (update_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_BF16) SHIFT(float, bf16);
  else if (update_dtype == FE_DTYPE_BF16 && out_dtype == FE_DTYPE_F32) SHIFT(bf16, float);
  else if (update_dtype == FE_DTYPE_BF16 && out_dtype == FE_DTYPE_BF16) SHIFT(bf16, bf16);
#undef SHIFT
#undef SHIFT_V
  return rc ? rc : fe_last_error();
}

// ---------------------------------------------------------------------------
// wkv_decay: out[t, c] = exp(-exp(base[c] + sum_j tanh(low[t, j]) up[j, c])), all 32-bit
// ---------------------------------------------------------------------------
// A block takes TOKENS tokens and 256 / SPLIT channels; SPLIT groups of threads share the rank and
// meet in shared memory in a fixed order.
template <int TOKENS, int SPLIT>
__global__ void __launch_bounds__(256)
wkv_decay_kernel(const float* __restrict__ low, const float* __restrict__ up, const float* __restrict__ base,
                 float* __restrict__ out, int n_tokens, int rank, int channels) {
  constexpr int CHANNELS = 256 / SPLIT;
  extern __shared__ __align__(16) float th[];       // [rank][TOKENS], then the groups' sums
  pdl_trigger();
  pdl_wait();
  const int t0 = blockIdx.y * TOKENS, count = min(TOKENS, n_tokens - t0);
  for (int i = threadIdx.x; i < rank * TOKENS; i += blockDim.x) {
    const int j = i / TOKENS, t = i - j * TOKENS;
    th[i] = t < count ? tanhf(low[(size_t)(t0 + t) * rank + j]) : 0.f;
  }
  __syncthreads();
  const int g = threadIdx.x / CHANNELS, x = threadIdx.x - g * CHANNELS, c = blockIdx.x * CHANNELS + x;
  float acc[TOKENS];
#pragma unroll
  for (int t = 0; t < TOKENS; ++t) acc[t] = 0.f;
  if (c < channels) {
#pragma unroll 8
    for (int j = g; j < rank; j += SPLIT) {
      const float u = up[(size_t)j * channels + c];
#pragma unroll
      for (int t = 0; t < TOKENS; t += 4) {
        const float4 a = *reinterpret_cast<const float4*>(th + j * TOKENS + t);
        acc[t] = fmaf(a.x, u, acc[t]), acc[t + 1] = fmaf(a.y, u, acc[t + 1]);
        acc[t + 2] = fmaf(a.z, u, acc[t + 2]), acc[t + 3] = fmaf(a.w, u, acc[t + 3]);
      }
    }
  }
  const float b0 = c < channels ? base[c] : 0.f;
  if constexpr (SPLIT == 1) {
    if (c < channels)
#pragma unroll
      for (int t = 0; t < TOKENS; ++t)
        if (t < count) out[(size_t)(t0 + t) * channels + c] = expf(-expf(b0 + acc[t]));
  } else {
    float* part = th + rank * TOKENS;               // [SPLIT][TOKENS][CHANNELS]
#pragma unroll
    for (int t = 0; t < TOKENS; ++t) part[(g * TOKENS + t) * CHANNELS + x] = acc[t];
    __syncthreads();
    if (c >= channels) return;
    for (int t = g; t < count; t += SPLIT) {
      float sum = 0.f;
#pragma unroll
      for (int k = 0; k < SPLIT; ++k) sum += part[(k * TOKENS + t) * CHANNELS + x];
      out[(size_t)(t0 + t) * channels + c] = expf(-expf(b0 + sum));
    }
  }
}

template <int TOKENS, int SPLIT>
static int launch_decay(const float* low, const float* up, const float* base, float* out, int n_tokens, int rank, int channels,
                        cudaStream_t stream) {
  const size_t smem = sizeof(float) * TOKENS * ((size_t)rank + (SPLIT > 1 ? 256 : 0));
  const int channels_a_block = 256 / SPLIT, blocks_y = (n_tokens + TOKENS - 1) / TOKENS;
  if (smem > 200 * 1024 || blocks_y > 65535) return FE_ERR_TOO_LARGE;
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(wkv_decay_kernel<TOKENS, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  return fe_launch_dependent(wkv_decay_kernel<TOKENS, SPLIT>, dim3((channels + channels_a_block - 1) / channels_a_block, blocks_y),
                             dim3(256), smem, stream, low, up, base, out, n_tokens, rank, channels);
}

FE_EXPORT int fe_wkv_decay(const float* low, const float* up, const float* base, float* out, int n_tokens, int rank,
                           int channels, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (rank < 1 || channels < 1) return FE_ERR_BAD_SHAPE;
  const int rc = n_tokens > 256 && rank <= 1024 ? launch_decay<32, 1>(low, up, base, out, n_tokens, rank, channels, stream)
                                                : launch_decay<8, 8>(low, up, base, out, n_tokens, rank, channels, stream);
  return rc ? rc : fe_last_error();
}

// ---------------------------------------------------------------------------
// the recurrence
// ---------------------------------------------------------------------------
struct Wkv {
  const float *r, *k, *f;   // [tokens, heads * dk], f the decay
  long long ld;
  const float* u;           // [heads, dk]
  // chunk-parallel scratch
  float* o_local;           // [tokens, heads, dv]
  float* qb;                // [tokens, heads, dk]
  float* local;             // [slots, heads, dk, dv]: a chunk's end state from a zero start, then (scan) its start state
  float* decay;             // [slots, heads, dk]

  static constexpr int VECS = 3, SCALARS = 1, EXTRA = 0;
  static constexpr bool SCORES = false, NORMALISER = false;

  __device__ __forceinline__ float* column(const StateRun& p, int slot, int head, int col, size_t* step) const {
    *step = p.dv;
    return p.state + ((size_t)slot * p.heads + head) * p.dk * p.dv + col;
  }
  __device__ __forceinline__ void begin(const StateRun&, int, int, float*) const {}
  __device__ __forceinline__ void end(const StateRun&, int, int, const float*) const {}
  // how much of its own value a token's output gets: sum_d r_d u_d k_d
  __device__ __forceinline__ float bonus(const StateRun& p, int head, int token) const {
    const size_t at = (size_t)token * ld + (size_t)head * p.dk;
    float b = 0.f;
    for (int d = threadIdx.x & 31; d < p.dk; d += 32) b = fmaf(r[at + d] * u[head * p.dk + d], k[at + d], b);
    return warp_sum(b);
  }
  __device__ __forceinline__ void stage(const StateRun& p, int head, int first, int nt, float* vec, int pitch, float* sc) const {
    for (int i = threadIdx.x; i < nt * p.dk; i += blockDim.x) {
      const int t = i / p.dk, d = i - t * p.dk;
      const size_t at = (size_t)(first + t) * ld + (size_t)head * p.dk + d;
      float* dst = vec + t * VECS * pitch + d;
      dst[0] = r[at], dst[pitch] = k[at], dst[2 * pitch] = f[at];
    }
    for (int t = threadIdx.x >> 5; t < nt; t += blockDim.x >> 5) {
      const float b = bonus(p, head, first + t);
      if ((threadIdx.x & 31) == 0) sc[t] = b;
    }
  }
  template <int KPT>
  __device__ __forceinline__ float step(float (&S)[KPT], const float* vec, int pitch, const float* sc, float value, int s, int ds) const {
    const float *rs = vec + s, *ks = rs + pitch, *fs = ks + pitch;
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
      acc = fmaf(S[i], rs[i * ds], acc);
      S[i] = fmaf(fs[i * ds], S[i], ks[i * ds] * value);
    }
    return fmaf(sc[0], value, sr_column_sum(acc, ds));
  }
  __device__ __forceinline__ float scale(const float*, const float*, int) const { return 1.f; }

  __device__ __forceinline__ Rows queries(const StateRun& p, int head, const ChunkAt& at) const {
    return Rows{qb + ((size_t)at.first * p.heads + head) * p.dk, (long long)p.heads * p.dk};
  }
  __device__ __forceinline__ float query_mul() const { return 1.f; }
  __device__ __forceinline__ Rows starts(const StateRun& p, int head, const ChunkAt& at) const {
    return Rows{local + ((size_t)at.slot * p.heads + head) * p.dk * p.dv, p.dv};
  }
  __device__ __forceinline__ Rows locals(const StateRun& p, int head, const ChunkAt& at) const {
    return Rows{o_local + ((size_t)at.first * p.heads + head) * p.dv, (long long)p.heads * p.dv};
  }
  __device__ __forceinline__ void out_begin(const StateRun&, int, const ChunkAt& at, double*, double*, float* ea, float*) const {
    for (int t = threadIdx.x; t < SR_LONG; t += 32) ea[t] = t < at.count ? 1.f : 0.f;
  }
};

// One chunk from a zero state.  A thread keeps rows s * KPT .. of two columns, so that a token's
// decays, keys and receptances are read 16 bytes at a time and serve both; rows past dk are padded
// with zeros, and a pitch of KPT + 4 keeps a column's lanes in different banks.  Tokens come in
// stretches of SR_CHUNK, the next one on its way into the other half of the buffers meanwhile.
#define WL_KPT 16
#define WL_KP (WL_KPT + 4)
__global__ void __launch_bounds__(512) wkv_local_kernel(const Wkv m, const StateRun p, int splits, int cols, int wide) {
  extern __shared__ __align__(16) float smem[];
  pdl_trigger();
  pdl_wait();
  ChunkAt at;
  if (!sr_locate(p, &at)) return;
  const int head = blockIdx.x / splits, split = blockIdx.x - head * splits;
  const int dk = p.dk, dv = p.dv, ds = p.ds, pitch = ds * WL_KP, tid = threadIdx.x;
  const int part = SR_CHUNK * pitch, half_size = 3 * part + SR_CHUNK * cols;
  float* bonus = smem + 2 * half_size;       // [SR_CHUNK]
  float* bs = bonus + SR_CHUNK;              // [dk]: the product of the decays so far
  const int v = tid / ds, s = tid - v * ds, half = cols >> 1, col0 = split * cols;
  const int lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
  const bool live = v < half;
  uint64_t S0[WL_KPT / 2], S1[WL_KPT / 2];      // neighbouring rows in pairs
#pragma unroll
  for (int i = 0; i < WL_KPT / 2; ++i) S0[i] = S1[i] = 0;
  for (int i = tid; i < 2 * half_size; i += blockDim.x) smem[i] = 0.f;
  for (int d = tid; d < dk; d += blockDim.x) bs[d] = 1.f;
  __syncthreads();
  const size_t head_at = (size_t)head * dk;
  // half of the buffers: decays [SR_CHUNK][ds][WL_KP], receptances, keys, values [SR_CHUNK][cols]
  auto fetch = [&](int c0, float* buf) {
    const int nt = min(SR_CHUNK, at.count - c0), first = at.first + c0;
    for (int t = warp; t < nt; t += warps) {
      const size_t row = (size_t)(first + t) * m.ld + head_at;
      float* dst = buf + t * pitch;
      if (wide) {
        for (int d = 4 * lane; d < dk; d += 128) {
          float* to = dst + (d / WL_KPT) * WL_KP + d % WL_KPT;
          sr_copy16(to, m.f + row + d), sr_copy16(to + part, m.r + row + d), sr_copy16(to + 2 * part, m.k + row + d);
        }
      } else {
        for (int d = lane; d < dk; d += 32) {
          float* to = dst + (d / WL_KPT) * WL_KP + d % WL_KPT;
          sr_copy4(to, m.f + row + d), sr_copy4(to + part, m.r + row + d), sr_copy4(to + 2 * part, m.k + row + d);
        }
      }
      const float* value = p.v + (size_t)(first + t) * p.v_ld + (size_t)head * dv + col0;
      for (int c = lane; c < cols && col0 + c < dv; c += 32) sr_copy4(buf + 3 * part + t * cols + c, value + c);
    }
    sr_copy_commit();
  };
  fetch(0, smem);
  int turn = 0;
  for (int c0 = 0; c0 < at.count; c0 += SR_CHUNK, turn ^= 1) {
    const int nt = min(SR_CHUNK, at.count - c0), first = at.first + c0;
    float* buf = smem + turn * half_size;
    const float *fs = buf, *rs = buf + part, *ks = rs + part, *vs = ks + part;
    sr_copy_wait<0>();
    __syncthreads();
    if (c0 + SR_CHUNK < at.count) fetch(c0 + SR_CHUNK, smem + (turn ^ 1) * half_size);
    for (int t = warp; t < nt; t += warps) {
      float b = 0.f;
      for (int d = lane; d < dk; d += 32) {
        const int i = t * pitch + (d / WL_KPT) * WL_KP + d % WL_KPT;
        b = fmaf(rs[i] * m.u[head_at + d], ks[i], b);
      }
      b = warp_sum(b);
      if (lane == 0) bonus[t] = b;
    }
    if (split == 0) {
      for (int d = tid; d < dk; d += blockDim.x) {
        const int from = (d / WL_KPT) * WL_KP + d % WL_KPT;
        float b = bs[d];
        float* dst = m.qb + ((size_t)first * p.heads + head) * dk + d;
#pragma unroll 4
        for (int t = 0; t < nt; ++t) {
          dst[(size_t)t * p.heads * dk] = rs[t * pitch + from] * b;
          b *= fs[t * pitch + from];
        }
        bs[d] = b;
      }
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float v0 = live ? vs[t * cols + v] : 0.f, v1 = live ? vs[t * cols + half + v] : 0.f;
      const ulonglong2* f2 = reinterpret_cast<const ulonglong2*>(fs + t * pitch + s * WL_KP);
      const ulonglong2* r2 = reinterpret_cast<const ulonglong2*>(rs + t * pitch + s * WL_KP);
      const ulonglong2* k2 = reinterpret_cast<const ulonglong2*>(ks + t * pitch + s * WL_KP);
      const uint64_t vv0 = sr_pair(v0, v0), vv1 = sr_pair(v1, v1);
      uint64_t acc0 = 0, acc1 = 0;
#pragma unroll
      for (int i = 0; i < WL_KPT / 4; ++i) {
        const ulonglong2 f = f2[i], r = r2[i], k = k2[i];
        acc0 = sr_fma2(S0[2 * i], r.x, acc0);
        acc1 = sr_fma2(S1[2 * i], r.x, acc1);
        S0[2 * i] = sr_fma2(f.x, S0[2 * i], sr_mul2(k.x, vv0));
        S1[2 * i] = sr_fma2(f.x, S1[2 * i], sr_mul2(k.x, vv1));
        acc0 = sr_fma2(S0[2 * i + 1], r.y, acc0);
        acc1 = sr_fma2(S1[2 * i + 1], r.y, acc1);
        S0[2 * i + 1] = sr_fma2(f.y, S0[2 * i + 1], sr_mul2(k.y, vv0));
        S1[2 * i + 1] = sr_fma2(f.y, S1[2 * i + 1], sr_mul2(k.y, vv1));
      }
      const float2 sum0 = sr_unpair(acc0), sum1 = sr_unpair(acc1);
      const float a0 = sr_column_sum(sum0.x + sum0.y, ds), a1 = sr_column_sum(sum1.x + sum1.y, ds);
      if (live && s == 0) {
        float* dst = m.o_local + ((size_t)(first + t) * p.heads + head) * dv + col0;
        if (col0 + v < dv) dst[v] = fmaf(bonus[t], v0, a0);
        if (col0 + half + v < dv) dst[half + v] = fmaf(bonus[t], v1, a1);
      }
    }
  }
  const size_t cell = (size_t)at.slot * p.heads + head;
#pragma unroll
  for (int i = 0; i < WL_KPT; ++i) {
    const int d = s * WL_KPT + i;
    if (!live || d >= dk) continue;
    float* dst = m.local + (cell * dk + d) * dv + col0;
    const float2 x0 = sr_unpair(S0[i / 2]), x1 = sr_unpair(S1[i / 2]);
    if (col0 + v < dv) dst[v] = i & 1 ? x0.y : x0.x;
    if (col0 + half + v < dv) dst[half + v] = i & 1 ? x1.y : x1.x;
  }
  if (split == 0)
    for (int d = tid; d < dk; d += blockDim.x) m.decay[cell * dk + d] = bs[d];
}

// One thread per state element walks an entry's chunks: every chunk's start state (in place of its
// local end state) and the request's state row after the last.
__global__ void __launch_bounds__(256) wkv_scan_kernel(const Wkv m, const StateRun p, int* status) {
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
  const int cell = blockIdx.z * blockDim.x + threadIdx.x;
  if (cell >= p.dk * p.dv) return;
  const int chunks = (count + SR_LONG - 1) / SR_LONG;
  const size_t base = (size_t)sr_slot(first, entry, 0) * p.heads + head, size = (size_t)p.dk * p.dv;
  float* st = p.state + ((size_t)slot * p.heads + head) * size + cell;
  float* local = m.local + base * size + cell;
  const float* decay = m.decay + base * p.dk + cell / p.dv;
  const size_t stride = (size_t)p.heads * size, dstride = (size_t)p.heads * p.dk;
  float state = *st;
  for (int c0 = 0; c0 < chunks; c0 += 8) {           // eight chunks' terms are fetched before any is replaced
    float add[8], keep[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const bool has = c0 + j < chunks;
      add[j] = has ? local[(size_t)(c0 + j) * stride] : 0.f;
      keep[j] = has ? decay[(size_t)(c0 + j) * dstride] : 1.f;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c0 + j < chunks) {
        local[(size_t)(c0 + j) * stride] = state;
        state = fmaf(keep[j], state, add[j]);
      }
    }
  }
  *st = state;
}

// Threads per column, columns per block and column blocks of wkv_local; false: sizes it does not take.
static bool wkv_local_shape(int dk, int dv, int* ds, int* cols, int* splits) {
  *ds = 1;
  while (*ds * WL_KPT < dk) *ds <<= 1;
  if (*ds > 16) return false;
  *splits = 1;
  while ((((dv + *splits - 1) / *splits + 1) / 2) * *ds > 512) *splits <<= 1;
  *cols = ((dv + *splits - 1) / *splits + 1) / 2 * 2;
  return true;
}

// 32-bit floats of scratch for a step of `tokens` tokens in `entries` entries, for entries of
// SR_LONG_FROM tokens or more to run chunk by chunk (0: these sizes are walked whatever their
// length) and for the walk in stretches of columns.
FE_EXPORT long long fe_wkv_scratch(int tokens, int entries, int heads, int dk, int max_new) {
  const int dv = dk;
  int ds, cols, splits;
  long long need = walk_in_stretches(dk, dv, 0) ? (long long)tokens * heads * dv : 0;
  if (max_new < SR_LONG_FROM || !chunk_takes(dk, dv, false) || !wkv_local_shape(dk, dv, &ds, &cols, &splits)) return need;
  return need + (long long)tokens * heads * (dk + dv) + sr_slots(tokens, entries) * heads * ((long long)dk * dv + dk);
}

FE_EXPORT int fe_wkv(const float* r, const float* k, const float* v, const float* decay, long long ld, const float* u,
                     const float* norm_w, const float* gate, long long gate_ld, float eps, float* state, int state_rows,
                     const int* slots, const int* cu_tokens, void* out, int out_dtype, int entries, int heads, int dk,
                     int tokens, int max_new, float* scratch, int* status, cudaStream_t stream) {
  if (entries <= 0 || tokens <= 0) return 0;
  if (heads < 1 || dk < 1 || heads > 65535 || entries > 65535) return FE_ERR_BAD_SHAPE;
  const int dv = dk;
  StateRun p{state, state_rows, slots, cu_tokens, heads, dk, dv, 0, v, ld, norm_w, dv, gate, gate_ld, 0, eps, out, nullptr, 0};
  Wkv m{r, k, decay, ld, u, nullptr, nullptr, nullptr, nullptr};
  if (walk_in_stretches(dk, dv, 0)) {
    p.raw = scratch;
    scratch = scratch ? scratch + (size_t)tokens * heads * dv : nullptr;
  }
  int ds, cols, splits;
  const bool chunked = max_new >= SR_LONG_FROM && scratch != nullptr && chunk_takes(dk, dv, false) && wkv_local_shape(dk, dv, &ds, &cols, &splits);
  if (chunked) p.long_from = SR_LONG_FROM;
  int rc = launch_walk(m, p, out_dtype, entries, tokens, status, stream);
  if (rc || !chunked) return rc ? rc : fe_last_error();
  const int chunks = (max_new + SR_LONG - 1) / SR_LONG;
  if (chunks > 65535) return FE_ERR_TOO_LARGE;
  m.o_local = scratch;
  m.qb = m.o_local + (size_t)tokens * heads * dv;
  m.local = m.qb + (size_t)tokens * heads * dk;
  m.decay = m.local + (size_t)sr_slots(tokens, entries) * heads * dk * dv;
  p.ds = ds;
  const int threads = (cols / 2 * ds + 31) / 32 * 32;
  const size_t smem = sizeof(float) * ((size_t)SR_CHUNK * (2 * (3 * ds * WL_KP + cols) + 1) + dk);
  const int wide = dk % 4 == 0 && ld % 4 == 0 && (((uintptr_t)r | (uintptr_t)k | (uintptr_t)decay) & 15) == 0;
  if (smem > 48 * 1024) cudaFuncSetAttribute(wkv_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  rc = fe_launch_dependent(wkv_local_kernel, dim3(heads * splits, entries, chunks), dim3(threads), smem, stream, m, p, splits, cols, wide);
  if (rc) return rc;
  rc = fe_launch_dependent(wkv_scan_kernel, dim3(heads, entries, (dk * dv + 255) / 256), dim3(256), 0, stream, m, p, status);
  if (rc) return rc;
  rc = launch_out(m, p, out_dtype, entries, chunks, stream);
  return rc ? rc : fe_last_error();
}

// Tokens from which on an entry of these recurrences runs chunk by chunk.
FE_EXPORT int fe_state_long_from() { return SR_LONG_FROM; }
