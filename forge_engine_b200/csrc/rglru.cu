// The real-gated linear recurrent unit of Griffin's recurrent block, with the short convolution in front
// of it and the gate behind it.  Per channel c of `width`, in part b of `part` channels:
//
//     u_t = conv(x)_t + conv_b          causal, over time
//     r = sigmoid(R_b u_b + br),  i = sigmoid(I_b u_b + bi)
//     log a = rate r  (rate = -strength softplus(lam), at most 0),  a = exp(log a)
//     S_t = a S_(t-1) + sqrt(1 - a^2) i u_t
//     out_t = S_t gelu_tanh(y_t)
//
// x and y are 32-bit sums of the projection.  Everything here is 32-bit; with bfloat16 gate matrices u
// enters their product as the sum of two bfloat16 numbers (the rounded one and the rounded remainder).
//
//   rglru_gates   tiles of 64 tokens of the step (whatever entries they belong to) x 64 channels of one
//                 part: convolution, both products, gates, and the recurrence from zero inside the tile.
//                 Leaves, per token, h (the state if the tile had started from zero, or the entry began
//                 inside it) and the product of the a since then, so that S = h + prod * S_in.
//   rglru_chain   walks an entry's tiles with one multiply-add each, leaves every tile's incoming state,
//                 the request's new state, and the convolution's last inputs.
//   rglru_out     S and the output of every token.
//   rglru_step    steps in which every entry brings one token (bfloat16): all of it in one launch.  The
//                 blocks of a part form a cluster; each convolves its own channels, moves their history
//                 on and hands them to the others through shared memory.
#include <cooperative_groups.h>

#include "mma_sync.cuh"

namespace cg = cooperative_groups;

struct Rglru {
  const float* proj;        // [tokens, ld]: y from column y_off, x from x_off
  long long ld;
  int y_off, x_off;
  const float* conv_w;      // [taps, width], the last tap weighs the token itself
  const float* conv_b;      // [width]
  int taps;
  const void *wr, *wi;      // [blocks, part, part], a gate's row is the output channel
  const float *y_bias, *x_bias;     // [width]: of the projection, not yet in proj
  const float *br, *bi, *rate;      // [width]
  float* state;             // [rows, width]
  float* conv_state;        // [rows, taps - 1, width], oldest first
  int state_rows;
  const int *slots, *cu_tokens, *token_entry;
  int width, part, n_tokens, n_entries;
  float *h, *prod;          // [tokens, width]
  float *carry, *init;      // [tiles, width]: state before a tile's first token; [entries, width]: before an entry's
  void* out;                // [tokens, width]
};

#define RG_KC 64            // channels of a part taken at a time
#define RG_WP (RG_KC + 8)   // pitch of a bfloat16 tile
#define RG_FP (RG_KC + 4)   // pitch of a 32-bit tile

__device__ __forceinline__ float rg_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rg_reciprocal(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rg_sigmoid(float z) { return rg_reciprocal(1.f + rg_exp2(-1.4426950408889634f * z)); }
__device__ __forceinline__ float rg_gelu(float z) {
  // 0.5 (1 + tanh(t)) = sigmoid(2 t)
  return z * rg_sigmoid(1.5957691216057308f * (z + 0.044715f * z * z * z));
}
// 1 - e^(-x) for x >= 0, given e = e^(-x): near zero by the power series, whose terms keep the digits
// that the subtraction would lose
__device__ __forceinline__ float rg_one_minus_exp(float x, float e) {
  float s = fmaf(x, -1.f / 7.f, 1.f);
  s = fmaf(-x * (1.f / 6.f), s, 1.f);
  s = fmaf(-x * (1.f / 5.f), s, 1.f);
  s = fmaf(-x * (1.f / 4.f), s, 1.f);
  s = fmaf(-x * (1.f / 3.f), s, 1.f);
  s = fmaf(-x * (1.f / 2.f), s, 1.f);
  return x < 0.25f ? x * s : 1.f - e;
}
__device__ __forceinline__ float rg_sqrt(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// a and the input's factor sqrt(1 - a^2) i from the gates' sums
__device__ __forceinline__ void rg_gates(float zr, float zi, float rate, float* a, float* scale) {
  const float log_a = rate * rg_sigmoid(zr);
  *a = expf(log_a);
  *scale = rg_sqrt(rg_one_minus_exp(-2.f * log_a, *a * *a)) * rg_sigmoid(zi);
}
__device__ __forceinline__ void rg_copy4(void* dst, const void* src, bool valid) {
  const int bytes = valid ? 4 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(bytes) : "memory");
}

// Rows n0 .. n0 + rows - 1 of one part's gate matrix, columns k0 .. k0 + cols - 1, into dst[row * pitch + col];
// zero outside the matrix.  `cols` is a multiple of 8.
__device__ __forceinline__ void rg_load_weight(bf16* dst, int pitch, const bf16* w, int part, int n0, int rows, int k0, int cols) {
  if (part % 8 == 0) {
    const int pieces = cols >> 3;
    for (int i = threadIdx.x; i < rows * pieces; i += blockDim.x) {
      const int n = i / pieces, k = (i - n * pieces) * 8;
      const bool has = n0 + n < part && k0 + k < part;
      cp_async16(dst + n * pitch + k, has ? w + (size_t)(n0 + n) * part + k0 + k : w, has);
    }
    return;
  }
  for (int i = threadIdx.x; i < rows * cols; i += blockDim.x) {
    const int n = i / cols, k = i - n * cols;
    dst[n * pitch + k] = n0 + n < part && k0 + k < part ? w[(size_t)(n0 + n) * part + k0 + k] : __float2bfloat16_rn(0.f);
  }
}
__device__ __forceinline__ void rg_load_weight(float* dst, int pitch, const float* w, int part, int n0, int rows, int k0, int cols) {
  if (part % 4 == 0) {
    const int pieces = cols >> 2;
    for (int i = threadIdx.x; i < rows * pieces; i += blockDim.x) {
      const int n = i / pieces, k = (i - n * pieces) * 4;
      const bool has = n0 + n < part && k0 + k < part;
      cp_async16(dst + n * pitch + k, has ? w + (size_t)(n0 + n) * part + k0 + k : w, has);
    }
    return;
  }
  for (int i = threadIdx.x; i < rows * cols; i += blockDim.x) {
    const int n = i / cols, k = i - n * cols;
    const bool has = n0 + n < part && k0 + k < part;
    rg_copy4(dst + n * pitch + k, has ? w + (size_t)(n0 + n) * part + k0 + k : w, has);
  }
}

// ---------------------------------------------------------------------------
// rglru_gates
// ---------------------------------------------------------------------------
#define RG_RM 64            // tokens of a tile
#define RG_NC RG_KC         // channels of a block's tile: one chunk of its part
#define RG_THREADS 256

template <typename TW>
struct RgShape {
  static constexpr bool MMA = sizeof(TW) == 2;
  static constexpr int BLOCKS = MMA ? 3 : 1;                                           // an SM's share, by registers
  static constexpr int WPITCH = MMA ? RG_WP : RG_FP;
  static constexpr size_t W_BYTES = sizeof(TW) * 2 * RG_NC * WPITCH;                   // both gates, one stage
  static constexpr size_t A_BYTES = MMA ? sizeof(bf16) * 2 * RG_RM * RG_WP : sizeof(float) * RG_RM * RG_FP;
  static_assert(2 * W_BYTES >= sizeof(float) * 2 * RG_RM * (RG_NC + 1), "the gates' sums lie over the matrices' stages");
  static size_t bytes(int taps) { return A_BYTES + 2 * W_BYTES + sizeof(float) * (RG_RM + taps - 1) * RG_KC; }
};

// TAPS: 4, or 0 for any number.
template <typename TW, int TAPS>
__global__ void __launch_bounds__(RG_THREADS, RgShape<TW>::BLOCKS) rglru_gates_kernel(const Rglru p, int* status) {
  using Shape = RgShape<TW>;
  constexpr int NC = RG_NC;
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ int since[RG_RM], slot_of[RG_RM];       // tokens since the entry's first; the request's row (-1: none)
  __shared__ float seg_h[4][NC], seg_p[4][NC];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n0 = blockIdx.x * NC, block = blockIdx.y, t0 = blockIdx.z * RG_RM;
  const int part = p.part, taps = TAPS > 0 ? TAPS : p.taps, back = taps - 1;
  const int rows = min(RG_RM, p.n_tokens - t0);
  unsigned char* as = raw;                                                     // u: hi and lo [RM][RG_WP], or 32-bit [RM][RG_FP]
  TW* ws = reinterpret_cast<TW*>(raw + Shape::A_BYTES);                        // [2 stages][2 gates][NC][pitch]
  float* xs = reinterpret_cast<float*>(raw + Shape::A_BYTES + 2 * Shape::W_BYTES);       // [RM + back][KC]
  const TW* wr = (const TW*)p.wr + (size_t)block * part * part;
  const TW* wi = (const TW*)p.wi + (size_t)block * part * part;
  const int x0 = block * part;                       // the part's first channel
  const bool wide = part % 4 == 0 && p.ld % 4 == 0 && p.x_off % 4 == 0 && ((uintptr_t)p.proj & 15) == 0;
  auto load = [&](int k0, int stage) {
    TW* w = ws + stage * 2 * NC * Shape::WPITCH;
    rg_load_weight(w, Shape::WPITCH, wr, part, n0, NC, k0, RG_KC);
    rg_load_weight(w + NC * Shape::WPITCH, Shape::WPITCH, wi, part, n0, NC, k0, RG_KC);
    float* x = xs;
    const float* src = p.proj + p.x_off + x0 + k0;
    if (wide) {
      for (int i = tid; i < (RG_RM + back) * (RG_KC / 4); i += RG_THREADS) {
        const int r = i / (RG_KC / 4), c = (i - r * (RG_KC / 4)) * 4, t = t0 + r - back;
        const bool has = t >= 0 && t < p.n_tokens && k0 + c < part;
        cp_async16(x + r * RG_KC + c, has ? src + (size_t)t * p.ld + c : p.proj, has);
      }
    } else {
      for (int i = tid; i < (RG_RM + back) * RG_KC; i += RG_THREADS) {
        const int r = i / RG_KC, c = i - r * RG_KC, t = t0 + r - back;
        const bool has = t >= 0 && t < p.n_tokens && k0 + c < part;
        rg_copy4(x + r * RG_KC + c, has ? src + (size_t)t * p.ld + c : p.proj, has);
      }
    }
    cp_commit();
  };
  // the part's chunks of channels, the block's own last: its u then stays where the products read it
  const int chunks = (part + RG_KC - 1) / RG_KC, mine = n0 / RG_KC;
  auto chunk_at = [&](int i) { return (i + mine + 1 < chunks ? i + mine + 1 : i + mine + 1 - chunks) * RG_KC; };
  load(chunk_at(0), 0);
  int n = 1 << 30;                                   // past the last token: as if far inside an entry
  if (tid < RG_RM) {
    int s = -1;
    if (tid < rows) {
      const int entry = p.token_entry[t0 + tid];
      n = t0 + tid - p.cu_tokens[entry];
      s = p.slots[entry];
      if (s < 0 || s >= p.state_rows) {
        atomicOr(status, FE_STATUS_BAD_PAGE);
        s = -1;
      }
    }
    since[tid] = n, slot_of[tid] = s;
  }
  const bool edge = __syncthreads_or(n < back);      // some tokens' taps reach into a request's state
  const bool begins = __syncthreads_or(n == 0);      // an entry begins in this tile

  // products: a warp takes 16 tokens x 32 channels of both gates; 32-bit: a thread 4 x 4
  float acc[2][4][4];
#pragma unroll
  for (int g = 0; g < 2; ++g)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[g][j][e] = 0.f;
  const int rw = warp & 3, cw = warp >> 2;
  const int fr = (tid & 15) * 4, fc = tid >> 4;      // 32-bit: rows fr .. fr + 3, channels fc + NC / 4 * e
  // the convolution: a thread takes two channels of PER neighbouring tokens
  constexpr int PER = RG_RM / (RG_THREADS / 32);
  const int c2 = lane * 2, r0 = warp * PER;

  for (int i = 0; i < chunks; ++i) {
    const int k0 = chunk_at(i), stage = i & 1;
    cp_wait<0>();
    __syncthreads();
    {
      const float* x = xs + c2;
      const int ch = x0 + k0 + c2;
      const bool live0 = k0 + c2 < part, live1 = k0 + c2 + 1 < part;
      auto put = [&](int r, float u0, float u1) {
        if constexpr (Shape::MMA) {
          unsigned h, l;
          split2(u0, u1, h, l);
          bf16* hi = reinterpret_cast<bf16*>(as) + r * RG_WP + c2;
          *reinterpret_cast<unsigned*>(hi) = h;
          *reinterpret_cast<unsigned*>(hi + RG_RM * RG_WP) = l;
        } else {
          *reinterpret_cast<float2*>(reinterpret_cast<float*>(as) + r * RG_FP + c2) = make_float2(u0, u1);
        }
      };
      if (TAPS > 0 && !edge) {
        // every tap inside the step: the projection's bias goes through the taps' sum
        float w0[TAPS > 0 ? TAPS : 1], w1[TAPS > 0 ? TAPS : 1], b0 = 0.f, b1 = 0.f;
        float2 in[TAPS > 0 ? TAPS : 1];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          w0[j] = live0 ? p.conv_w[(size_t)j * p.width + ch] : 0.f;
          w1[j] = live1 ? p.conv_w[(size_t)j * p.width + ch + 1] : 0.f;
          b0 += w0[j], b1 += w1[j];
          in[j] = *reinterpret_cast<const float2*>(x + (r0 + (j < TAPS - 1 ? j : 0)) * RG_KC);
        }
        b0 = live0 ? fmaf(b0, p.x_bias[ch], p.conv_b[ch]) : 0.f;
        b1 = live1 ? fmaf(b1, p.x_bias[ch + 1], p.conv_b[ch + 1]) : 0.f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
          in[TAPS > 0 ? TAPS - 1 : 0] = *reinterpret_cast<const float2*>(x + (r0 + i + back) * RG_KC);
          float u0 = b0, u1 = b1;
#pragma unroll
          for (int j = 0; j < TAPS; ++j) u0 = fmaf(w0[j], in[j].x, u0), u1 = fmaf(w1[j], in[j].y, u1);
          put(r0 + i, u0, u1);
#pragma unroll
          for (int j = 0; j + 1 < TAPS; ++j) in[j] = in[j + 1];
        }
      } else {
        for (int r = r0; r < r0 + PER; ++r) {
          float u[2] = {0.f, 0.f};
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            if (!(e == 0 ? live0 : live1)) continue;
            const float bias = p.x_bias[ch + e];
            u[e] = p.conv_b[ch + e];
            for (int j = 0; j < taps; ++j) {
              // index into (the state's rows, the entry's rows)
              const int at = since[r] < back ? since[r] + j : back;
              float v = 0.f;
              if (at >= back) v = x[(r + j) * RG_KC + e] + bias;
              else if (slot_of[r] >= 0) v = p.conv_state[((size_t)slot_of[r] * back + at) * p.width + ch + e];
              u[e] = fmaf(p.conv_w[(size_t)j * p.width + ch + e], v, u[e]);
            }
          }
          put(r, u[0], u[1]);
        }
      }
    }
    __syncthreads();
    if (i + 1 < chunks) load(chunk_at(i + 1), stage ^ 1);      // while the products run
    const TW* w = ws + stage * 2 * NC * Shape::WPITCH;
    if constexpr (Shape::MMA) {
      const bf16* hi = reinterpret_cast<const bf16*>(as);
#pragma unroll
      for (int kk = 0; kk < RG_KC / 16; ++kk) {
        unsigned ah[4], al[4];
        const int a_at = (rw * 16 + (lane & 15)) * RG_WP + kk * 16 + (lane >> 4) * 8;
        ldsm4(ah[0], ah[1], ah[2], ah[3], hi + a_at);
        ldsm4(al[0], al[1], al[2], al[3], hi + RG_RM * RG_WP + a_at);
#pragma unroll
        for (int g = 0; g < 2; ++g) {
#pragma unroll
          for (int j = 0; j < 4; j += 2) {
            unsigned b0, b1, b2, b3;
            ldsm4(b0, b1, b2, b3, reinterpret_cast<const bf16*>(w) + (g * NC + cw * 32 + (j + (lane >> 4)) * 8 + (lane & 7)) * RG_WP +
                                      kk * 16 + ((lane >> 3) & 1) * 8);
            mma16816(acc[g][j], ah, b0, b1);
            mma16816(acc[g][j + 1], ah, b2, b3);
            mma16816(acc[g][j], al, b0, b1);
            mma16816(acc[g][j + 1], al, b2, b3);
          }
        }
      }
    } else {
      const float* u = reinterpret_cast<const float*>(as);
      for (int k = 0; k < RG_KC; ++k) {
        float a[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) a[e] = u[(fr + e) * RG_FP + k];
#pragma unroll
        for (int g = 0; g < 2; ++g)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float b = reinterpret_cast<const float*>(w)[(g * NC + fc + NC / 4 * j) * RG_FP + k];
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[g][j][e] = fmaf(a[e], b, acc[g][j][e]);
          }
      }
    }
  }
  __syncthreads();

  // the sums of both gates, [gate][RM][NC + 1], over the matrices
  float* gates = reinterpret_cast<float*>(ws);
  constexpr int GP = NC + 1;
#pragma unroll
  for (int g = 0; g < 2; ++g)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        int r, c;
        if constexpr (Shape::MMA) r = rw * 16 + (lane >> 2) + 8 * (e >> 1), c = cw * 32 + j * 8 + (lane & 3) * 2 + (e & 1);
        else r = fr + e, c = fc + NC / 4 * j;
        gates[(g * RG_RM + r) * GP + c] = acc[g][j][e];
      }
  __syncthreads();

  // the recurrence from zero: a thread takes one channel of 16 tokens, then learns what the tile's
  // earlier tokens leave (unless an entry begins in between)
  const int c = tid % NC, seg = tid / NC, r_from = seg * 16;
  const bool live = n0 + c < part;
  const int ch = live ? x0 + n0 + c : x0;
  const float br = p.br[ch], bi = p.bi[ch], rate = p.rate[ch];
  float h[16], prod[16];
  int fresh = 16;                        // the segment's first row that begins an entry
  {
    float s = 0.f, q = 1.f;
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      const int r = r_from + i;
      float a, scale;
      rg_gates(gates[r * GP + c] + br, gates[(RG_RM + r) * GP + c] + bi, rate, &a, &scale);
      if (begins && since[r] == 0) {
        s = 0.f, q = 1.f;
        fresh = min(fresh, i);
      }
      float u;
      if constexpr (Shape::MMA) {
        const bf16* hi = reinterpret_cast<const bf16*>(as) + r * RG_WP + c;
        u = __bfloat162float(hi[0]) + __bfloat162float(hi[RG_RM * RG_WP]);
      } else {
        u = reinterpret_cast<const float*>(as)[r * RG_FP + c];
      }
      s = fmaf(a, s, scale * u);
      q *= a;
      h[i] = s, prod[i] = q;
    }
    seg_h[seg][c] = s, seg_p[seg][c] = q;
  }
  __syncthreads();
  if (!live) return;
  float h_in = 0.f, p_in = 1.f;
  for (int s = 0; s < seg; ++s) {
    bool cut = false;
    if (begins)
      for (int r = s * 16; r < s * 16 + 16; ++r) cut = cut || since[r] == 0;
    h_in = cut ? seg_h[s][c] : fmaf(seg_p[s][c], h_in, seg_h[s][c]);
    p_in = cut ? seg_p[s][c] : seg_p[s][c] * p_in;
  }
  float *hp = p.h + (size_t)(t0 + r_from) * p.width + ch, *pp = p.prod + (size_t)(t0 + r_from) * p.width + ch;
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    if (r_from + i < rows) {
      const bool joined = i < fresh;
      hp[(size_t)i * p.width] = joined ? fmaf(prod[i], h_in, h[i]) : h[i];
      pp[(size_t)i * p.width] = joined ? prod[i] * p_in : prod[i];
    }
  }
}

// ---------------------------------------------------------------------------
// rglru_chain: a thread per entry and channel
// ---------------------------------------------------------------------------
__global__ void __launch_bounds__(64) rglru_chain_kernel(const Rglru p) {
  pdl_trigger();
  pdl_wait();
  const int entry = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int first = p.cu_tokens[entry], end = p.cu_tokens[entry + 1], slot = p.slots[entry];
  if (c >= p.width || end <= first || slot < 0 || slot >= p.state_rows) return;
  float* cell = p.state + (size_t)slot * p.width + c;
  float s = *cell;
  p.init[(size_t)entry * p.width + c] = s;
  const int k_from = first / RG_RM, k_to = (end - 1) / RG_RM;
  for (int k0 = k_from; k0 <= k_to; k0 += 16) {
    float h[16], a[16];
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      const bool has = k0 + j <= k_to;
      const size_t at = (size_t)(has ? min((k0 + j + 1) * RG_RM, end) - 1 : first) * p.width + c;
      h[j] = has ? p.h[at] : 0.f;
      a[j] = has ? p.prod[at] : 1.f;
    }
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      s = fmaf(a[j], s, h[j]);
      if (k0 + j < k_to) p.carry[(size_t)(k0 + j + 1) * p.width + c] = s;
    }
  }
  *cell = s;
  // the last taps - 1 of (the state's inputs, the step's): a row is read before it is overwritten
  const int back = p.taps - 1, count = end - first;
  float* st = p.conv_state + (size_t)slot * back * p.width + c;
  for (int k = 0; k < back; ++k) {
    const int at = count + k;
    st[(size_t)k * p.width] = at < back ? st[(size_t)at * p.width] : p.proj[(size_t)(first + at - back) * p.ld + p.x_off + c] + p.x_bias[c];
  }
}

// ---------------------------------------------------------------------------
// rglru_out: S and the output, V neighbouring channels a thread
// ---------------------------------------------------------------------------
template <typename TO, int V>
__global__ void __launch_bounds__(256) rglru_out_kernel(const Rglru p) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= p.width) return;
  const int entry = p.token_entry[t], tile = t / RG_RM;
  const float* in = p.cu_tokens[entry] >= tile * RG_RM ? p.init + (size_t)entry * p.width : p.carry + (size_t)tile * p.width;
  const size_t at = (size_t)t * p.width + c;
  const float* yp = p.proj + (size_t)t * p.ld + p.y_off + c;
  float h[V], a[V], s[V], y[V], b[V];
  if constexpr (V == 4) load4(p.h + at, h), load4(p.prod + at, a), load4(in + c, s), load4(yp, y), load4(p.y_bias + c, b);
  else h[0] = p.h[at], a[0] = p.prod[at], s[0] = in[c], y[0] = yp[0], b[0] = p.y_bias[c];
#pragma unroll
  for (int e = 0; e < V; ++e) h[e] = fmaf(a[e], s[e], h[e]) * rg_gelu(y[e] + b[e]);
  if constexpr (V == 4) store4((TO*)p.out + at, h);
  else ((TO*)p.out)[at] = from_float<TO>(h[0]);
}

// ---------------------------------------------------------------------------
// rglru_step
// ---------------------------------------------------------------------------
#define RG_SM 16            // entries of a tile
#define RG_HIST 7           // earlier inputs of the convolution held in registers

template <int NC>
static size_t rg_step_smem(int part) {
  const size_t pitch = (size_t)(part + 15) / 16 * 16 + 8;
  return sizeof(bf16) * (2 * NC + 2 * RG_SM) * pitch + sizeof(float) * 3 * RG_SM * (NC + 1);
}

template <typename TO, int NC>
__global__ void __launch_bounds__(4 * NC) rglru_step_kernel(const Rglru p, int* status) {
  extern __shared__ __align__(16) unsigned char raw[];
  cg::cluster_group cluster = cg::this_cluster();
  constexpr int THREADS = 4 * NC, GP = NC + 1;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n0 = blockIdx.x * NC, block = blockIdx.y, t0 = blockIdx.z * RG_SM;
  const int part = p.part, k_all = (part + 15) / 16 * 16, pitch = k_all + 8, back = p.taps - 1;
  const int rows = min(RG_SM, p.n_tokens - t0);
  bf16* ws = reinterpret_cast<bf16*>(raw);            // [2 gates][NC][pitch]
  bf16* hi = ws + 2 * NC * pitch;                     // [SM][pitch]: u of the whole part, rounded; then the remainders
  float* us = reinterpret_cast<float*>(hi + 2 * RG_SM * pitch);      // [SM][GP]: u of the block's own channels
  float* gates = us + RG_SM * GP;                     // [2][SM][GP]
  pdl_trigger();
  // the gate matrices are nobody's output: on their way before the kernels ahead have finished
  rg_load_weight(ws, pitch, (const bf16*)p.wr + (size_t)block * part * part, part, n0, NC, 0, k_all);
  rg_load_weight(ws + NC * pitch, pitch, (const bf16*)p.wi + (size_t)block * part * part, part, n0, NC, 0, k_all);
  cp_commit();
  for (int i = tid; i < RG_SM * pitch / 4; i += THREADS) reinterpret_cast<uint4*>(hi)[i] = make_uint4(0u, 0u, 0u, 0u);
  auto arrived = cluster.barrier_arrive();            // this block is there and its tiles are zero
  // a thread's four (entry, channel) places; what they need is fetched before anything waits for it
  const int x0 = block * part, cols = min(NC, part - n0);
  const int peers = (int)cluster.num_blocks();
  const int c = tid % NC, ch = x0 + n0 + c;
  const bool has = c < cols;
  float u[4], y[4], before[4], fresh[4], hist[4][RG_HIST], taps_w[RG_HIST + 1];
  int slot[4];
  const float br = has ? p.br[ch] : 0.f, bi = has ? p.bi[ch] : 0.f, rate = has ? p.rate[ch] : 0.f;
  const float conv_b = has ? p.conv_b[ch] : 0.f, x_bias = has ? p.x_bias[ch] : 0.f, y_bias = has ? p.y_bias[ch] : 0.f;
#pragma unroll
  for (int j = 0; j < RG_HIST + 1; ++j) taps_w[j] = has && j <= back ? p.conv_w[(size_t)j * p.width + ch] : 0.f;
  pdl_wait();
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int r = tid / NC + 4 * k;
    slot[k] = has && r < rows ? p.slots[t0 + r] : -1;
    if (has && r < rows && (slot[k] < 0 || slot[k] >= p.state_rows)) {
      atomicOr(status, FE_STATUS_BAD_PAGE);
      slot[k] = -1;
    }
    u[k] = y[k] = before[k] = fresh[k] = 0.f;
    if (slot[k] < 0) continue;
    const float* row = p.proj + (size_t)(t0 + r) * p.ld + ch;
    fresh[k] = row[p.x_off] + x_bias, y[k] = row[p.y_off] + y_bias;
    before[k] = p.state[(size_t)slot[k] * p.width + ch];
    if (back <= RG_HIST) {
#pragma unroll
      for (int j = 0; j < RG_HIST; ++j)
        hist[k][j] = j < back ? p.conv_state[((size_t)slot[k] * back + j) * p.width + ch] : 0.f;
    }
  }
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int r = tid / NC + 4 * k;
    if (slot[k] >= 0) {
      // the oldest input leaves the history, the others move up
      float* st = p.conv_state + (size_t)slot[k] * back * p.width + ch;
      u[k] = conv_b;
      if (back <= RG_HIST) {
#pragma unroll
        for (int j = 0; j < RG_HIST; ++j) {
          if (j < back) {
            u[k] = fmaf(taps_w[j], hist[k][j], u[k]);
            if (j > 0) st[(size_t)(j - 1) * p.width] = hist[k][j];
          }
        }
#pragma unroll
        for (int j = 0; j < RG_HIST + 1; ++j)
          if (j == back) u[k] = fmaf(taps_w[j], fresh[k], u[k]);
      } else {
        for (int j = 0; j < back; ++j) {
          const float v = st[(size_t)j * p.width];
          u[k] = fmaf(p.conv_w[(size_t)j * p.width + ch], v, u[k]);
          if (j > 0) st[(size_t)(j - 1) * p.width] = v;
        }
        u[k] = fmaf(p.conv_w[(size_t)back * p.width + ch], fresh[k], u[k]);
      }
      if (back > 0) st[(size_t)(back - 1) * p.width] = fresh[k];
    }
    us[r * GP + c] = u[k];
  }
  __syncthreads();
  cluster.barrier_wait(std::move(arrived));           // every block of the cluster is there
  // channels of a part in pairs: n0 is even
  for (int i = tid; i < rows * (NC / 2); i += THREADS) {
    const int r = i / (NC / 2), c2 = (i - r * (NC / 2)) * 2;
    if (c2 >= cols) continue;
    unsigned h, l;
    split2(us[r * GP + c2], us[r * GP + c2 + 1], h, l);     // past the last channel: zero
    const int at = r * pitch + n0 + c2;
    for (int peer = 0; peer < peers; ++peer) {
      bf16* dst = cluster.map_shared_rank(hi, peer);
      *reinterpret_cast<unsigned*>(dst + at) = h;
      *reinterpret_cast<unsigned*>(dst + RG_SM * pitch + at) = l;
    }
  }
  cp_wait<0>();
  __syncthreads();
  cluster.sync();                                     // the whole part's u is in place
  {
    // a warp takes 16 channels of one gate
    const int g = warp / (NC / 16), c0 = (warp - g * (NC / 16)) * 16;
    float acc[4][4] = {};        // products of the rounded numbers, then of the remainders
#pragma unroll 4
    for (int kk = 0; kk < k_all / 16; ++kk) {
      unsigned ah[4], al[4], b0, b1, b2, b3;
      const int a_at = (lane & 15) * pitch + kk * 16 + (lane >> 4) * 8;
      ldsm4(ah[0], ah[1], ah[2], ah[3], hi + a_at);
      ldsm4(al[0], al[1], al[2], al[3], hi + RG_SM * pitch + a_at);
      ldsm4(b0, b1, b2, b3, ws + (g * NC + c0 + (lane >> 4) * 8 + (lane & 7)) * pitch + kk * 16 + ((lane >> 3) & 1) * 8);
      mma16816(acc[0], ah, b0, b1);
      mma16816(acc[1], ah, b2, b3);
      mma16816(acc[2], al, b0, b1);
      mma16816(acc[3], al, b2, b3);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        gates[(g * RG_SM + (lane >> 2) + 8 * (e >> 1)) * GP + c0 + j * 8 + (lane & 3) * 2 + (e & 1)] = acc[j][e] + acc[2 + j][e];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    if (slot[k] < 0) continue;
    const int r = tid / NC + 4 * k;
    float a, scale;
    rg_gates(gates[r * GP + c] + br, gates[(RG_SM + r) * GP + c] + bi, rate, &a, &scale);
    const float s = fmaf(a, before[k], scale * u[k]);
    p.state[(size_t)slot[k] * p.width + ch] = s;
    ((TO*)p.out)[(size_t)(t0 + r) * p.width + ch] = from_float<TO>(s * rg_gelu(y[k]));
  }
}

// ---------------------------------------------------------------------------
// launchers
// ---------------------------------------------------------------------------
template <typename TO, int NC>
static int rg_launch_step(const Rglru& p, int* status, cudaStream_t stream) {
  const size_t smem = rg_step_smem<NC>(p.part);
  if (smem > 48 * 1024) cudaFuncSetAttribute(rglru_step_kernel<TO, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  const unsigned tiles = (unsigned)((p.part + NC - 1) / NC);
  return fe_launch_dependent_shaped(rglru_step_kernel<TO, NC>, dim3(tiles, p.width / p.part, (p.n_tokens + RG_SM - 1) / RG_SM), dim3(4 * NC),
                                    smem, stream, dim3(tiles, 1, 1), p, status);
}

// Channels of a block of rglru_step for parts of this size: at most 8 blocks share a part; 0: not taken.
static int rg_step_cols(int part) {
  if (part <= 8 * 32 && rg_step_smem<32>(part) <= 200 * 1024) return 32;
  if (part <= 8 * 64 && rg_step_smem<64>(part) <= 200 * 1024) return 64;
  return 0;
}

template <typename TW, int TAPS>
static int rg_launch_gates(const Rglru& p, int* status, cudaStream_t stream) {
  using Shape = RgShape<TW>;
  const size_t smem = Shape::bytes(p.taps);
  if (smem > 220 * 1024) return FE_ERR_TOO_LARGE;
  cudaFuncSetAttribute(rglru_gates_kernel<TW, TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  const dim3 grid((p.part + RG_NC - 1) / RG_NC, p.width / p.part, (p.n_tokens + RG_RM - 1) / RG_RM);
  return fe_launch_dependent(rglru_gates_kernel<TW, TAPS>, grid, dim3(RG_THREADS), smem, stream, p, status);
}

// Whether a step in which every entry brings one token is one launch.
FE_EXPORT int fe_rglru_one_launch(int part, int weight_dtype) { return weight_dtype == FE_DTYPE_BF16 && rg_step_cols(part) > 0; }

// Floats of scratch a step of these sizes needs otherwise.
FE_EXPORT long long fe_rglru_scratch(int tokens, int entries, int width) {
  return (2LL * tokens + (tokens + RG_RM - 1) / RG_RM + 1 + entries) * ((width + 3) / 4 * 4);
}

FE_EXPORT int fe_rglru(const float* proj, long long ld, int y_off, int x_off, const float* conv_w, const float* conv_b, int taps,
                       const void* wr, const void* wi, int weight_dtype, const float* y_bias, const float* x_bias, const float* br, const float* bi, const float* rate,
                       float* state, float* conv_state, int state_rows, const int* slots, const int* cu_tokens,
                       const int* token_entry, void* out, int out_dtype, int width, int part, int tokens, int entries, int max_new,
                       float* scratch, int* status, cudaStream_t stream) {
  if (tokens <= 0 || entries <= 0) return 0;
  if (taps < 1 || width < 1 || part < 1 || width % part || width / part > 65535 || entries > 65535 || (taps > 1 && conv_state == nullptr))
    return FE_ERR_BAD_SHAPE;
  if ((tokens + RG_SM - 1) / RG_SM > 65535) return FE_ERR_TOO_LARGE;
  if (((uintptr_t)wr | (uintptr_t)wi) & 15) return FE_ERR_BAD_ALIGN;
  Rglru p{proj, ld, y_off, x_off, conv_w, conv_b, taps, wr, wi, y_bias, x_bias, br, bi, rate, state, conv_state, state_rows, slots, cu_tokens,
          token_entry, width, part, tokens, entries, nullptr, nullptr, nullptr, nullptr, out};
  int rc = FE_ERR_BAD_DTYPE;
  if (max_new == 1 && tokens == entries && fe_rglru_one_launch(part, weight_dtype)) {
    const int cols = rg_step_cols(part);
    if (out_dtype == FE_DTYPE_BF16) rc = cols == 32 ? rg_launch_step<bf16, 32>(p, status, stream) : rg_launch_step<bf16, 64>(p, status, stream);
    else if (out_dtype == FE_DTYPE_F32) rc = cols == 32 ? rg_launch_step<float, 32>(p, status, stream) : rg_launch_step<float, 64>(p, status, stream);
    return rc ? rc : fe_last_error();
  }
  if (scratch == nullptr) return FE_ERR_BAD_SHAPE;
  const size_t tiles = (size_t)(tokens + RG_RM - 1) / RG_RM, pitch = (size_t)width;
  p.h = scratch;
  p.prod = p.h + (size_t)tokens * pitch;
  p.carry = p.prod + (size_t)tokens * pitch;
  p.init = p.carry + (tiles + 1) * pitch;
  if (weight_dtype == FE_DTYPE_BF16) rc = taps == 4 ? rg_launch_gates<bf16, 4>(p, status, stream) : rg_launch_gates<bf16, 0>(p, status, stream);
  else if (weight_dtype == FE_DTYPE_F32) rc = taps == 4 ? rg_launch_gates<float, 4>(p, status, stream) : rg_launch_gates<float, 0>(p, status, stream);
  if (rc) return rc;
  rc = fe_launch_dependent(rglru_chain_kernel, dim3((width + 63) / 64, entries), dim3(64), 0, stream, p);
  if (rc) return rc;
  const bool wide = width % 4 == 0 && ld % 4 == 0 && y_off % 4 == 0 && (((uintptr_t)proj | (uintptr_t)scratch | (uintptr_t)out | (uintptr_t)y_bias) & 15) == 0;
  const int per = wide ? 4 : 1;
  int threads = 32;
  while (threads < 256 && threads * per < width) threads <<= 1;
  const dim3 grid(tokens, (width + threads * per - 1) / (threads * per));
  if (out_dtype == FE_DTYPE_BF16)
    rc = wide ? fe_launch_dependent(rglru_out_kernel<bf16, 4>, grid, dim3(threads), 0, stream, p) : fe_launch_dependent(rglru_out_kernel<bf16, 1>, grid, dim3(threads), 0, stream, p);
  else if (out_dtype == FE_DTYPE_F32)
    rc = wide ? fe_launch_dependent(rglru_out_kernel<float, 4>, grid, dim3(threads), 0, stream, p) : fe_launch_dependent(rglru_out_kernel<float, 1>, grid, dim3(threads), 0, stream, p);
  else
    rc = FE_ERR_BAD_DTYPE;
  return rc ? rc : fe_last_error();
}
