// Embedding gather, fused residual-add + RMSNorm, SiLU*mul.
//
// Upstream counterparts: nn.Embedding (src/forge_engine/qwen3.py:325), the fused
// residual RMSNorm (src/forge_engine/_triton_kernels.py:32-58; plain form
// src/forge_engine/kernels/__init__.py:12-26) and F.silu(gate) * up
// (src/forge_engine/qwen3.py:227).  The residual stream is kept in 32-bit.
#include "common.cuh"

// ---------------------------------------------------------------------------
// embedding: residual[n, c, :] = float(table[ids[n], :]) * scale for each of `copies` streams;
// with a table of learned positions, row positions[n] of it is added (unscaled, in 32-bit)
// ---------------------------------------------------------------------------
template <typename T>
__global__ void embedding_kernel(const int* __restrict__ ids, const T* __restrict__ table,
                                 float* __restrict__ out, int hidden, int vocab, float scale, int copies,
                                 const int* __restrict__ positions, const T* __restrict__ pos_table, int pos_rows,
                                 int* status) {
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  const int id = ids[row];
  float* dst = out + (size_t)row * copies * hidden;
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) atomicOr(status, FE_STATUS_BAD_TOKEN);
    for (int i = threadIdx.x; i < copies * hidden; i += blockDim.x) dst[i] = 0.f;
    return;
  }
  const T* src = table + (size_t)id * hidden;
  const T* place = nullptr;
  if (pos_table != nullptr) {
    const int pos = positions[row];
    if (pos < 0 || pos >= pos_rows) {
      if (threadIdx.x == 0) atomicOr(status, FE_STATUS_BAD_POSITION);
    } else {
      place = pos_table + (size_t)pos * hidden;
    }
  }
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    float v = scale == 1.f ? to_float(src[i]) : to_float(src[i]) * scale;
    if (place != nullptr) v += to_float(place[i]);
    for (int c = 0; c < copies; ++c) dst[(size_t)c * hidden + i] = v;
  }
}

FE_EXPORT int fe_embedding(const int* ids, const void* table, int table_dtype, float* out,
                           int n, int hidden, int vocab, float scale, int copies, const int* positions,
                           const void* pos_table, int pos_rows, int* status, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (copies < 1) return FE_ERR_BAD_SHAPE;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == FE_DTYPE_F32)
    return fe_launch_dependent(embedding_kernel<float>, dim3(n), dim3(threads), 0, stream, ids, (const float*)table, out, hidden, vocab, scale, copies, positions, (const float*)pos_table, pos_rows, status);
  else if (table_dtype == FE_DTYPE_BF16)
    return fe_launch_dependent(embedding_kernel<bf16>, dim3(n), dim3(threads), 0, stream, ids, (const bf16*)table, out, hidden, vocab, scale, copies, positions, (const bf16*)pos_table, pos_rows, status);
  else
    return FE_ERR_BAD_DTYPE;
  return fe_last_error();
}

// ---------------------------------------------------------------------------
// x = residual[src] + update[src] (+ shift[src], rows shift_stride apart; 0: one vector for all rows);  residual[src] = x (optional);
// out[r] = x * rsqrt(mean(x^2) + eps) * weight       -- all in 32-bit, one rounding
// src = row_map ? row_map[r] : r
// ---------------------------------------------------------------------------
template <typename TU, typename TO, int PER>
__global__ void add_rmsnorm_kernel(float* __restrict__ residual, const TU* __restrict__ update,
                                   const float* __restrict__ weight, TO* __restrict__ out,
                                   const int* __restrict__ row_map, const float* __restrict__ shift, long long shift_stride, int size, float eps,
                                   int write_residual) {
  // PER > 0: every thread keeps its PER elements (strided by blockDim) in registers between
  // the two passes; PER == 0: rows too long for that are read twice.
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x;
  const int src = row_map ? row_map[r] : r;
  float* res = residual + (size_t)src * size;
  const TU* upd = update ? update + (size_t)src * size : nullptr;
  TO* dst = out + (size_t)r * size;
  if (shift) shift += (size_t)src * shift_stride;
  float ss = 0.f;
  if constexpr (PER > 0) {
    float x[PER > 0 ? PER : 1];
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      x[j] = 0.f;
      if (i < size) {
        x[j] = res[i];
        if (upd) x[j] += to_float(upd[i]);
        if (shift) x[j] += shift[i];
        if (write_residual) res[i] = x[j];
        ss += x[j] * x[j];
      }
    }
    const float inv = rsqrtf(block_sum(ss, scratch) / (float)size + eps);
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < size) dst[i] = from_float<TO>(x[j] * inv * weight[i]);
    }
  } else {
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
      float x = res[i];
      if (upd) x += to_float(upd[i]);
      if (shift) x += shift[i];
      if (write_residual) res[i] = x;
      ss += x * x;
    }
    const float total = block_sum(ss, scratch);
    const float inv = rsqrtf(total / (float)size + eps);
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
      float x = res[i];
      if (upd && !write_residual) x += to_float(upd[i]);
      if (shift && !write_residual) x += shift[i];
      dst[i] = from_float<TO>(x * inv * weight[i]);
    }
  }
}

// Rows whose length is a multiple of 4 and at most 4 * 4 * 1024: a thread keeps up to PER
// groups of four neighbouring elements (16-byte loads of the residual), same arithmetic.
template <typename TU, typename TO, int PER>
__global__ void add_rmsnorm_vec_kernel(float* __restrict__ residual, const TU* __restrict__ update,
                                       const float* __restrict__ weight, TO* __restrict__ out,
                                       const int* __restrict__ row_map, const float* __restrict__ shift, long long shift_stride, int size, float eps,
                                       int write_residual) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x;
  const int src = row_map ? row_map[r] : r;
  float* res = residual + (size_t)src * size;
  const TU* upd = update ? update + (size_t)src * size : nullptr;
  TO* dst = out + (size_t)r * size;
  if (shift) shift += (size_t)src * shift_stride;
  const int groups = size >> 2;
  float x[PER][4];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int g = threadIdx.x + j * blockDim.x;
    if (g < groups) {
      load4(res + 4 * g, x[j]);
      if (upd) {
        float u[4];
        load4(upd + 4 * g, u);
#pragma unroll
        for (int e = 0; e < 4; ++e) x[j][e] += u[e];
      }
      if (shift) {
        float u[4];
        load4(shift + 4 * g, u);
#pragma unroll
        for (int e = 0; e < 4; ++e) x[j][e] += u[e];
      }
      if (write_residual) store4(res + 4 * g, x[j]);
#pragma unroll
      for (int e = 0; e < 4; ++e) ss += x[j][e] * x[j][e];
    }
  }
  const float inv = rsqrtf(block_sum(ss, scratch) / (float)size + eps);
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int g = threadIdx.x + j * blockDim.x;
    if (g < groups) {
      float w[4], y[4];
      load4(weight + 4 * g, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = x[j][e] * inv * w[e];
      store4(dst + 4 * g, y);
    }
  }
}

FE_EXPORT int fe_add_rmsnorm(float* residual, const void* update, int update_dtype,
                             const float* weight, void* out, int out_dtype, const int* row_map,
                             const float* shift, long long shift_stride, int rows, int size, float eps, int write_residual,
                             cudaStream_t stream) {
  if (rows <= 0) return 0;
  int rc = 0;
  const int update_bytes = update_dtype == FE_DTYPE_F32 ? 16 : 8, out_bytes = out_dtype == FE_DTYPE_F32 ? 16 : 8;
  if ((size % 4) == 0 && size <= 16384 && ((uintptr_t)residual % 16) == 0 && ((uintptr_t)weight % 16) == 0 &&
      ((uintptr_t)update % update_bytes) == 0 && ((uintptr_t)out % out_bytes) == 0 && ((uintptr_t)shift % 16) == 0 && (shift_stride % 4) == 0) {
    const int groups = size / 4;
    const int per = groups <= 1024 ? 1 : groups <= 2048 ? 2 : 4;
    const int vthreads = (((groups + per - 1) / per) + 31) / 32 * 32;
#define LAUNCH_VEC(TU, TO)                                                                                        \
    do {                                                                                                          \
      if (per == 1)                                                                                               \
        rc = fe_launch_dependent(add_rmsnorm_vec_kernel<TU, TO, 1>, dim3(rows), dim3(vthreads), 0, stream, residual, \
            (const TU*)update, weight, (TO*)out, row_map, shift, shift_stride, size, eps, write_residual);                             \
      else if (per == 2)                                                                                          \
        rc = fe_launch_dependent(add_rmsnorm_vec_kernel<TU, TO, 2>, dim3(rows), dim3(vthreads), 0, stream, residual, \
            (const TU*)update, weight, (TO*)out, row_map, shift, shift_stride, size, eps, write_residual);                             \
      else                                                                                                        \
        rc = fe_launch_dependent(add_rmsnorm_vec_kernel<TU, TO, 4>, dim3(rows), dim3(vthreads), 0, stream, residual, \
            (const TU*)update, weight, (TO*)out, row_map, shift, shift_stride, size, eps, write_residual);                             \
    } while (0)
    if (update_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_F32) LAUNCH_VEC(float, float);
    else if (update_dtype == FE_DTYPE_BF16 && out_dtype == FE_DTYPE_BF16) LAUNCH_VEC(bf16, bf16);
    else if (update_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_BF16) LAUNCH_VEC(float, bf16);
    else if (update_dtype == FE_DTYPE_BF16 && out_dtype == FE_DTYPE_F32) LAUNCH_VEC(bf16, float);
    else return FE_ERR_BAD_DTYPE;
#undef LAUNCH_VEC
    return rc ? rc : fe_last_error();
  }
  int threads = 32;
  while (threads < 512 && threads * 4 < size) threads <<= 1;
  const int per = (size + threads - 1) / threads;
#define LAUNCH(TU, TO)                                                                               \
  do {                                                                                               \
    if (per <= 4)                                                                                    \
      rc = fe_launch_dependent(add_rmsnorm_kernel<TU, TO, 4>, dim3(rows), dim3(threads), 0, stream, residual, (const TU*)update,      \
          weight, (TO*)out, row_map, shift, shift_stride, size, eps, write_residual);                                     \
    else if (per <= 16)                                                                              \
      rc = fe_launch_dependent(add_rmsnorm_kernel<TU, TO, 16>, dim3(rows), dim3(threads), 0, stream, residual, (const TU*)update,     \
          weight, (TO*)out, row_map, shift, shift_stride, size, eps, write_residual);                                     \
    else                                                                                             \
      rc = fe_launch_dependent(add_rmsnorm_kernel<TU, TO, 0>, dim3(rows), dim3(threads), 0, stream, residual, (const TU*)update,      \
          weight, (TO*)out, row_map, shift, shift_stride, size, eps, write_residual);                                     \
  } while (0)
  if (update_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_F32) LAUNCH(float, float);
  else if (update_dtype == FE_DTYPE_BF16 && out_dtype == FE_DTYPE_BF16) LAUNCH(bf16, bf16);
  else if (update_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_BF16) LAUNCH(float, bf16);
  else if (update_dtype == FE_DTYPE_BF16 && out_dtype == FE_DTYPE_F32) LAUNCH(bf16, float);
  else return FE_ERR_BAD_DTYPE;
#undef LAUNCH
  return rc ? rc : fe_last_error();
}

// ---------------------------------------------------------------------------
// out[n, i] = silu(gate_up[n, i]) * gate_up[n, inter + i]
// ---------------------------------------------------------------------------
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }

// block == 0: a row is [all gate | all up]; block == B > 0: a row alternates B gate
// features, B up features (the layout the fused projection kernels want).
__device__ __forceinline__ void silu_sources(int i, int inter, int block, int* gate_at, int* up_at) {
  if (block == 0) { *gate_at = i; *up_at = inter + i; }
  else { const int b = i / block; *gate_at = 2 * b * block + (i - b * block); *up_at = *gate_at + block; }
}

template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int inter, int block) {
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  const T* g = gate_up + (size_t)row * 2 * inter;
  T* o = out + (size_t)row * inter;
  const int i = blockIdx.y * blockDim.x + threadIdx.x;
  if (i >= inter) return;
  int ga, ua;
  silu_sources(i, inter, block, &ga, &ua);
  o[i] = from_float<T>(silu(to_float(g[ga])) * to_float(g[ua]));
}

template <typename T>
__global__ void silu_mul_vec8_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int inter, int block) {
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  const T* g = gate_up + (size_t)row * 2 * inter;
  T* o = out + (size_t)row * inter;
  const int i = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (i >= inter) return;
  int ga, ua;
  silu_sources(i, inter, block, &ga, &ua);   // block is a multiple of 8, so 8 features stay together
  float a[8], b[8];
  load8_streaming(g + ga, a);      // gate and up are read once: they need not stay in the caches
  load8_streaming(g + ua, b);
#pragma unroll
  for (int k = 0; k < 8; ++k) a[k] = silu(a[k]) * b[k];
  store8(o + i, a);
}

FE_EXPORT int fe_silu_mul(const void* gate_up, void* out, int dtype, int rows, int inter, int block,
                          cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (block < 0 || (block > 0 && (inter % block) != 0)) return FE_ERR_BAD_SHAPE;
  const bool vec = (inter % 8) == 0 && (block % 8) == 0 && ((uintptr_t)gate_up % 32) == 0 && ((uintptr_t)out % 32) == 0;
  const int threads = 256;
  const int per = vec ? 8 : 1;
  dim3 grid(rows, (inter + threads * per - 1) / (threads * per));
  if (grid.y > 65535) return FE_ERR_TOO_LARGE;
  if (dtype == FE_DTYPE_F32) {
    if (vec) return fe_launch_dependent(silu_mul_vec8_kernel<float>, grid, dim3(threads), 0, stream, (const float*)gate_up, (float*)out, inter, block);
    else return fe_launch_dependent(silu_mul_kernel<float>, grid, dim3(threads), 0, stream, (const float*)gate_up, (float*)out, inter, block);
  } else if (dtype == FE_DTYPE_BF16) {
    if (vec) return fe_launch_dependent(silu_mul_vec8_kernel<bf16>, grid, dim3(threads), 0, stream, (const bf16*)gate_up, (bf16*)out, inter, block);
    else return fe_launch_dependent(silu_mul_kernel<bf16>, grid, dim3(threads), 0, stream, (const bf16*)gate_up, (bf16*)out, inter, block);
  } else {
    return FE_ERR_BAD_DTYPE;
  }
  return fe_last_error();
}

// ---------------------------------------------------------------------------
// bias_xielu: out[n, i] = act(x[n, i] + bias[i]) with the activation
//   act(z) = a_pos z^2 + z / 2                 for z > 0
//            a_neg (exp(z) - 1 - z) + z / 2    for z <= 0
// taken in 32-bit of the projection's sums (bias 32-bit or null); one rounding on store.
// ---------------------------------------------------------------------------
template <typename TI, typename TO>
__global__ void __launch_bounds__(256)
bias_xielu_kernel(const TI* __restrict__ x, const float* __restrict__ bias, TO* __restrict__ out, long long total,
                  int width, float a_pos, float a_neg) {
  pdl_trigger();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    float z = to_float(x[i]);
    if (bias != nullptr) z += bias[(int)(i % width)];
    const float half = 0.5f * z;
    const float v = z > 0.f ? fmaf(a_pos * z, z, half) : fmaf(a_neg, expm1f(z) - z, half);
    out[i] = from_float<TO>(v);
  }
}

FE_EXPORT int fe_bias_xielu(const void* x, int x_dtype, const float* bias, void* out, int out_dtype, long long rows,
                            int width, float a_pos, float a_neg, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (width < 1) return FE_ERR_BAD_SHAPE;
  const long long total = rows * width;
  long long blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  int rc = FE_ERR_BAD_DTYPE;
#define XIELU(TI, TO) \
  rc = fe_launch_dependent(bias_xielu_kernel<TI, TO>, dim3((unsigned)blocks), dim3(256), 0, stream, (const TI*)x, bias, (TO*)out, total, width, a_pos, a_neg)
  if (x_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_F32) XIELU(float, float);
  else if (x_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_BF16) XIELU(float, bf16);
  else if (x_dtype == FE_DTYPE_BF16 && out_dtype == FE_DTYPE_BF16) XIELU(bf16, bf16);
#undef XIELU
  return rc ? rc : fe_last_error();
}

// ---------------------------------------------------------------------------
// bias_act: out[n, i] = act(x[n, i] + bias[i]) for an activation of one argument, taken in
// 32-bit of the projection's sums (bias 32-bit or null); one rounding on store.
//   act 0: the tanh form of GELU, 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3)))
//   act 1: the square of relu
// ---------------------------------------------------------------------------
template <typename TI, typename TO>
__global__ void __launch_bounds__(256)
bias_act_kernel(const TI* __restrict__ x, const float* __restrict__ bias, TO* __restrict__ out, long long total,
                int width, int act) {
  pdl_trigger();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    float z = to_float(x[i]);
    if (bias != nullptr) z += bias[(int)(i % width)];
    float v;
    if (act == 1) {
      const float r = fmaxf(z, 0.f);
      v = r * r;
    } else {
      v = 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    }
    out[i] = from_float<TO>(v);
  }
}

FE_EXPORT int fe_bias_act(const void* x, int x_dtype, const float* bias, void* out, int out_dtype, long long rows,
                          int width, int act, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (width < 1 || act < 0 || act > 1) return FE_ERR_BAD_SHAPE;
  const long long total = rows * width;
  long long blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  int rc = FE_ERR_BAD_DTYPE;
#define BIAS_ACT(TI, TO) \
  rc = fe_launch_dependent(bias_act_kernel<TI, TO>, dim3((unsigned)blocks), dim3(256), 0, stream, (const TI*)x, bias, (TO*)out, total, width, act)
  if (x_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_F32) BIAS_ACT(float, float);
  else if (x_dtype == FE_DTYPE_F32 && out_dtype == FE_DTYPE_BF16) BIAS_ACT(float, bf16);
  else if (x_dtype == FE_DTYPE_BF16 && out_dtype == FE_DTYPE_BF16) BIAS_ACT(bf16, bf16);
#undef BIAS_ACT
  return rc ? rc : fe_last_error();
}

// ---------------------------------------------------------------------------
// scale_cap: x <- x * scale, then (cap > 0) x <- cap * tanh(x / cap), in place on 32-bit values
// (a model's logits).
// ---------------------------------------------------------------------------
__global__ void __launch_bounds__(256) scale_cap_kernel(float* __restrict__ x, long long total, float scale, float cap) {
  pdl_trigger();
  pdl_wait();
  const float inv = cap > 0.f ? 1.f / cap : 0.f;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    float v = x[i] * scale;
    if (cap > 0.f) v = cap * tanhf(v * inv);
    x[i] = v;
  }
}

FE_EXPORT int fe_scale_cap(float* x, long long total, float scale, float cap, cudaStream_t stream) {
  if (total <= 0) return 0;
  long long blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  const int rc = fe_launch_dependent(scale_cap_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, x, total, scale, cap);
  return rc ? rc : fe_last_error();
}

// ---------------------------------------------------------------------------
// norm_pair: out = scale * (a / rms(a) * w_a + b / rms(b) * w_b) per row, rms over the row with
// eps inside the root; everything 32-bit (two mixers side by side, each normalised)
// ---------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
norm_pair_kernel(const float* __restrict__ a, const float* __restrict__ b, const float* __restrict__ w_a,
                 const float* __restrict__ w_b, float* __restrict__ out, int size, float eps, float scale) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const size_t at = (size_t)blockIdx.x * size;
  float sa = 0.f, sb = 0.f;
  for (int i = threadIdx.x; i < size; i += blockDim.x) {
    const float x = a[at + i], y = b[at + i];
    sa = fmaf(x, x, sa);
    sb = fmaf(y, y, sb);
  }
  const float ia = scale / sqrtf(block_sum(sa, scratch) / (float)size + eps);
  const float ib = scale / sqrtf(block_sum(sb, scratch) / (float)size + eps);
  for (int i = threadIdx.x; i < size; i += blockDim.x) out[at + i] = a[at + i] * ia * w_a[i] + b[at + i] * ib * w_b[i];
}

// The same for rows of up to 4,096 elements in fours: a thread keeps its four of both rows.
__global__ void __launch_bounds__(1024)
norm_pair_vec_kernel(const float* __restrict__ a, const float* __restrict__ b, const float* __restrict__ w_a,
                     const float* __restrict__ w_b, float* __restrict__ out, int size, float eps, float scale) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int i = 4 * threadIdx.x;
  const size_t at = (size_t)blockIdx.x * size + i;
  float x[4] = {0.f, 0.f, 0.f, 0.f}, y[4] = {0.f, 0.f, 0.f, 0.f}, u[4], v[4];
  float sa = 0.f, sb = 0.f;
  if (i < size) {
    load4(a + at, x), load4(b + at, y), load4(w_a + i, u), load4(w_b + i, v);
#pragma unroll
    for (int e = 0; e < 4; ++e) sa = fmaf(x[e], x[e], sa), sb = fmaf(y[e], y[e], sb);
  }
  const float ia = scale / sqrtf(block_sum(sa, scratch) / (float)size + eps);
  const float ib = scale / sqrtf(block_sum(sb, scratch) / (float)size + eps);
  if (i < size) {
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] = x[e] * ia * u[e] + y[e] * ib * v[e];
    store4(out + at, x);
  }
}

FE_EXPORT int fe_norm_pair(const float* a, const float* b, const float* w_a, const float* w_b, float* out, int rows, int size,
                           float eps, float scale, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (size < 1) return FE_ERR_BAD_SHAPE;
  if (size % 4 == 0 && size <= 4096 &&
      (((uintptr_t)a | (uintptr_t)b | (uintptr_t)w_a | (uintptr_t)w_b | (uintptr_t)out) & 15) == 0) {
    const int rc = fe_launch_dependent(norm_pair_vec_kernel, dim3(rows), dim3((size / 4 + 31) / 32 * 32), 0, stream, a, b, w_a, w_b, out, size, eps, scale);
    return rc ? rc : fe_last_error();
  }
  const int rc = fe_launch_dependent(norm_pair_kernel, dim3(rows), dim3(256), 0, stream, a, b, w_a, w_b, out, size, eps, scale);
  return rc ? rc : fe_last_error();
}

// ---------------------------------------------------------------------------
// weighted_sum: out = sa * a + sb * b, all 32-bit (two mixers side by side, added as they are)
// ---------------------------------------------------------------------------
template <int V>
__global__ void __launch_bounds__(256)
weighted_sum_kernel(const float* __restrict__ a, const float* __restrict__ b, float sa, float sb, float* __restrict__ out, long long count) {
  pdl_trigger();
  pdl_wait();
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (i >= count) return;
  if constexpr (V == 4) {
    float x[4], y[4];
    load4(a + i, x), load4(b + i, y);
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] = sa * x[e] + sb * y[e];
    store4(out + i, x);
  } else {
    out[i] = sa * a[i] + sb * b[i];
  }
}

FE_EXPORT int fe_weighted_sum(const float* a, const float* b, float sa, float sb, float* out, long long count, cudaStream_t stream) {
  if (count <= 0) return 0;
  const bool wide = count % 4 == 0 && (((uintptr_t)a | (uintptr_t)b | (uintptr_t)out) & 15) == 0;
  const long long blocks = (count / (wide ? 4 : 1) + 255) / 256;
  if (blocks > 0x7fffffffLL) return FE_ERR_TOO_LARGE;
  const int rc = wide ? fe_launch_dependent(weighted_sum_kernel<4>, dim3((unsigned)blocks), dim3(256), 0, stream, a, b, sa, sb, out, count)
                      : fe_launch_dependent(weighted_sum_kernel<1>, dim3((unsigned)blocks), dim3(256), 0, stream, a, b, sa, sb, out, count);
  return rc ? rc : fe_last_error();
}
