// Kernels of a real-gated linear recurrent unit: per channel c, with u the mixer's convolved input,
//
//   r = sigmoid(R u + b_r), i = sigmoid(I u + b_i)        R, I block-diagonal: B square blocks of n = W / B channels
//   a = exp(rate_c r)   (rate_c <= 0)
//   S <- a S + sqrt(1 - a^2) i u;   out = S gelu(y)        y the gate branch's projection, gelu in its tanh form
//
// S is one float per channel and request in the state slab.  Everything up to the product with gelu(y) is float32:
// u, both gates (their products with u as well), a, the step and S.
//
//   flint_rglru_gates   a and b = sqrt(1 - a^2) i u of every row, from u [T, W].  With bfloat16 blocks on the tensor
//                       cores: u is split into three bfloat16 numbers whose sum is u (8 bits of the significand each),
//                       so every product is exact and the sums are float32; otherwise on the float32 pipes.
//   flint_rglru_scan    S over the rows of every request, and out.  A request's rows are cut into chunks that are worked
//                       side by side: a first kernel leaves every chunk's product of a and its end state from zero,
//                       a second one starts each chunk from the state these give and walks it.
//   flint_rglru_step    a batch of single tokens in one launch: partial sums of the projection, convolution, gates,
//                       recurrence and the product with gelu(y).
//
// The convolution's last inputs lie in the request's state as a ring of `taps` rows (the input at position p in row
// p mod taps): one row more than are ever read, so that the row written for a token is none that its own
// convolution reads and several blocks may work on one token.
#include <math.h>
#include <stdarg.h>
#include "common.cuh"
#include "warp_mma.cuh"

using namespace flint;

namespace {

__device__ __forceinline__ float sigmoidf_(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float gelu_tanhf_(float x) {
  return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
}
// a and the input's factor for the gates' sums z_r and z_i
__device__ __forceinline__ void unit(float zr, float zi, float rate, float u, float& a, float& b) {
  const float la = rate * sigmoidf_(zr);
  a = expf(la);
  b = sqrtf(-expm1f(2.0f * la)) * sigmoidf_(zi) * u;       // 1 - a^2 without cancellation
}

// ------------------------------------------------------------------------------------------- gates, float32 pipes
constexpr int GM = 64, GN = 32, GK = 16;
template <typename TW>
__global__ void __launch_bounds__(256)
gates_simt_kernel(const float* __restrict__ u, const TW* __restrict__ wr, const float* __restrict__ br,
                  const TW* __restrict__ wi, const float* __restrict__ bi, const float* __restrict__ rate,
                  float* __restrict__ a_out, float* __restrict__ b_out, int T, int W, int n) {
  __shared__ float us[GK][GM + 4];
  __shared__ float rs[GK][GN + 4];
  __shared__ float is[GK][GN + 4];
  pdl_launch();
  pdl_wait();
  const int t0 = blockIdx.x * GM, o0 = blockIdx.y * GN, blk = blockIdx.z;
  const float* ub = u + (size_t)blk * n;
  const TW* wrb = wr + (size_t)blk * n * n;
  const TW* wib = wi + (size_t)blk * n * n;
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;       // 4 tokens by 2 outputs a thread
  float ar[4][2] = {}, ai[4][2] = {};
  for (int k0 = 0; k0 < n; k0 += GK) {
    for (int e = threadIdx.x; e < GM * GK; e += 256) {
      const int r = e / GK, k = e % GK;
      us[k][r] = (t0 + r < T && k0 + k < n) ? ub[(size_t)(t0 + r) * W + k0 + k] : 0.f;
    }
    for (int e = threadIdx.x; e < GN * GK; e += 256) {
      const int o = e / GK, k = e % GK;
      const bool ok = o0 + o < n && k0 + k < n;
      rs[k][o] = ok ? to_f32(wrb[(size_t)(o0 + o) * n + k0 + k]) : 0.f;
      is[k][o] = ok ? to_f32(wib[(size_t)(o0 + o) * n + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GK; ++k) {
      const float r0 = rs[k][2 * tx], r1 = rs[k][2 * tx + 1], i0 = is[k][2 * tx], i1 = is[k][2 * tx + 1];
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float x = us[k][4 * ty + q];
        ar[q][0] = fmaf(x, r0, ar[q][0]); ar[q][1] = fmaf(x, r1, ar[q][1]);
        ai[q][0] = fmaf(x, i0, ai[q][0]); ai[q][1] = fmaf(x, i1, ai[q][1]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int q = 0; q < 4; ++q)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int t = t0 + 4 * ty + q, o = o0 + 2 * tx + j;
      if (t >= T || o >= n) continue;
      const int c = blk * n + o;
      float a, b;
      unit(ar[q][j] + br[c], ai[q][j] + bi[c], rate[c], u[(size_t)t * W + c], a, b);
      a_out[(size_t)t * W + c] = a;
      b_out[(size_t)t * W + c] = b;
    }
}

// ------------------------------------------------------------------------------------------- gates, tensor cores
// A block takes 64 rows and 64 outputs of one diagonal block: four warps of 16 rows, both gates' sums in registers.
// Per stage of 32 channels u is split on the way into shared memory (three planes), R and I arrive by asynchronous
// copies.
constexpr int MM = 64, MN = 64, MK = 32, MS = MK + 8;
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__global__ void __launch_bounds__(128)
gates_mma_kernel(const float* __restrict__ u, const __nv_bfloat16* __restrict__ wr, const float* __restrict__ br,
                 const __nv_bfloat16* __restrict__ wi, const float* __restrict__ bi, const float* __restrict__ rate,
                 float* __restrict__ a_out, float* __restrict__ b_out, int T, int W, int n) {
  using flint_attn::ldsm4;
  using flint_attn::mma16816;
  __shared__ __align__(16) __nv_bfloat16 us[3][MM * MS];
  __shared__ __align__(16) __nv_bfloat16 ws[2][2][MN * MS];      // [stage][gate]
  pdl_launch();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = blockIdx.x * MM, o0 = blockIdx.y * MN, blk = blockIdx.z;
  const float* ub = u + (size_t)blk * n;
  auto fetch = [&](int k0, int st) {                             // weights are no kernel's output
    for (int c = tid; c < 2 * MN * (MK / 8); c += 128) {
      const int gate = c / (MN * (MK / 8)), x = c % (MN * (MK / 8)), o = x / (MK / 8), k = (x % (MK / 8)) * 8;
      const bool live = o0 + o < n && k0 + k < n;
      const __nv_bfloat16* src = (gate ? wi : wr) + ((size_t)blk * n + (live ? o0 + o : 0)) * n + (live ? k0 + k : 0);
      const uint32_t dst = smem_addr(&ws[st][gate][o * MS + k]);
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  pdl_wait();
  float4 ux[MM * MK / 4 / 128];                                  // this thread's pieces of the next stage of u
  auto load_u = [&](int k0) {
#pragma unroll
    for (int i = 0; i < MM * MK / 4 / 128; ++i) {
      const int c = tid + 128 * i, r = c / (MK / 4), k = (c % (MK / 4)) * 4;
      ux[i] = (t0 + r < T && k0 + k < n) ? *reinterpret_cast<const float4*>(ub + (size_t)(t0 + r) * W + k0 + k)
                                         : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  auto store_u = [&]() {
#pragma unroll
    for (int i = 0; i < MM * MK / 4 / 128; ++i) {
      const int c = tid + 128 * i, r = c / (MK / 4), k = (c % (MK / 4)) * 4;
      float v[4] = {ux[i].x, ux[i].y, ux[i].z, ux[i].w};
#pragma unroll
      for (int p = 0; p < 3; ++p) {
        __nv_bfloat16 h[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          h[e] = __float2bfloat16_rn(v[e]);
          v[e] -= __bfloat162float(h[e]);                        // exact: the rest fits the significand
        }
        *reinterpret_cast<uint2*>(&us[p][r * MS + k]) = *reinterpret_cast<const uint2*>(h);
      }
    }
  };
  float acc[2][MN / 8][4];
#pragma unroll
  for (int g = 0; g < 2; ++g)
#pragma unroll
    for (int i = 0; i < MN / 8; ++i) { acc[g][i][0] = acc[g][i][1] = acc[g][i][2] = acc[g][i][3] = 0.f; }
  load_u(0);
  int st = 0;
  for (int k0 = 0; k0 < n; k0 += MK, st ^= 1) {
    store_u();
    if (k0 + MK < n) {
      fetch(k0 + MK, st ^ 1);
      load_u(k0 + MK);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < MK; kk += 16) {
      uint32_t af[3][4];
#pragma unroll
      for (int p = 0; p < 3; ++p)
        ldsm4(smem_addr(&us[p][(warp * 16 + (lane & 15)) * MS + kk + (lane >> 4) * 8]), af[p][0], af[p][1], af[p][2], af[p][3]);
#pragma unroll
      for (int g = 0; g < 2; ++g)
#pragma unroll
        for (int nb = 0; nb < MN / 8; nb += 2) {
          uint32_t b0, b1, b2, b3;
          ldsm4(smem_addr(&ws[st][g][(nb * 8 + ((lane >> 4) << 3) + (lane & 7)) * MS + kk + ((lane >> 3) & 1) * 8]), b0, b1, b2, b3);
#pragma unroll
          for (int p = 2; p >= 0; --p) {                         // the smallest parts first
            mma16816(acc[g][nb], af[p][0], af[p][1], af[p][2], af[p][3], b0, b1);
            mma16816(acc[g][nb + 1], af[p][0], af[p][1], af[p][2], af[p][3], b2, b3);
          }
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = t0 + warp * 16 + (lane >> 2) + 8 * half;
    if (t >= T) continue;
#pragma unroll
    for (int nb = 0; nb < MN / 8; ++nb) {
      const int o = o0 + nb * 8 + 2 * (lane & 3);
      if (o >= n) continue;                                      // n is even
      const int c = blk * n + o;
      const float2 uu = *reinterpret_cast<const float2*>(u + (size_t)t * W + c);
      float2 a, b;
      unit(acc[0][nb][2 * half] + br[c], acc[1][nb][2 * half] + bi[c], rate[c], uu.x, a.x, b.x);
      unit(acc[0][nb][2 * half + 1] + br[c + 1], acc[1][nb][2 * half + 1] + bi[c + 1], rate[c + 1], uu.y, a.y, b.y);
      *reinterpret_cast<float2*>(a_out + (size_t)t * W + c) = a;
      *reinterpret_cast<float2*>(b_out + (size_t)t * W + c) = b;
    }
  }
}

// ------------------------------------------------------------------------------------------- the recurrence over rows
constexpr int CHUNK = 64;        // rows of a request worked by one block
constexpr int AHEAD = 8;         // rows whose operands are fetched together

// totals [n_seq, max_chunks + 1, 2, W]: entry 0 holds the request's state, entry c + 1 chunk c's product of a and its
// end state from zero.  Grid: (channel blocks, max_chunks, n_seq).
__global__ void rglru_totals_kernel(const float* __restrict__ a, const float* __restrict__ b, const int* __restrict__ slot,
                                    const int* __restrict__ seq_start, const float* __restrict__ state,
                                    long long state_stride, float* __restrict__ totals, int max_chunks, int W) {
  pdl_launch();
  pdl_wait();
  const int e = blockIdx.z, c = blockIdx.y, ch = blockIdx.x * blockDim.x + threadIdx.x;
  const int r0 = seq_start ? seq_start[e] : e, r1 = seq_start ? seq_start[e + 1] : e + 1;
  const int t0 = r0 + c * CHUNK, t1 = min(r1, t0 + CHUNK);
  if (ch >= W || t0 >= r1) return;
  float* mine = totals + (size_t)e * (max_chunks + 1) * 2 * W + ch;
  if (c == 0) mine[W] = state[(size_t)slot[r0] * state_stride + ch];
  if (t1 == r1) return;                       // the last chunk's totals are nobody's
  float A = 1.f, S = 0.f;
  for (int t = t0; t < t1; t += AHEAD) {      // a chunk that is not the last is whole
    float av[AHEAD], bv[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      av[i] = a[(size_t)(t + i) * W + ch];
      bv[i] = b[(size_t)(t + i) * W + ch];
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      A *= av[i];
      S = fmaf(av[i], S, bv[i]);
    }
  }
  mine[(size_t)(c + 1) * 2 * W] = A;
  mine[(size_t)(c + 1) * 2 * W + W] = S;
}

template <typename TO>
__global__ void rglru_walk_kernel(const float* __restrict__ a, const float* __restrict__ b, const float* __restrict__ y,
                                  long long y_stride, const int* __restrict__ slot, const int* __restrict__ seq_start,
                                  float* __restrict__ state, long long state_stride, const float* __restrict__ totals,
                                  int max_chunks, TO* __restrict__ out, int W) {
  pdl_launch();
  pdl_wait();
  const int e = blockIdx.z, c = blockIdx.y, ch = blockIdx.x * blockDim.x + threadIdx.x;
  const int r0 = seq_start ? seq_start[e] : e, r1 = seq_start ? seq_start[e + 1] : e + 1;
  const int t0 = r0 + c * CHUNK, t1 = min(r1, t0 + CHUNK);
  if (ch >= W || t0 >= r1) return;
  float* home = state + (size_t)slot[r0] * state_stride + ch;
  float S;
  if (totals) {
    const float* mine = totals + (size_t)e * (max_chunks + 1) * 2 * W + ch;
    S = mine[W];
#pragma unroll 8
    for (int k = 1; k <= c; ++k) S = fmaf(mine[(size_t)k * 2 * W], S, mine[(size_t)k * 2 * W + W]);
  } else {
    S = *home;
  }
  for (int t = t0; t < t1; t += AHEAD) {
    float av[AHEAD], bv[AHEAD], yv[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const bool in = t + i < t1;
      av[i] = in ? a[(size_t)(t + i) * W + ch] : 1.f;
      bv[i] = in ? b[(size_t)(t + i) * W + ch] : 0.f;
      yv[i] = in ? y[(size_t)(t + i) * y_stride + ch] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      S = fmaf(av[i], S, bv[i]);
      if (t + i < t1) out[(size_t)(t + i) * W + ch] = from_f32<TO>(S * gelu_tanhf_(yv[i]));
    }
  }
  if (t1 == r1) *home = S;
}

// ------------------------------------------------------------------------------------------- single tokens
// Block: SO outputs of one diagonal block for up to ST tokens.  The threads first form the convolved input of the
// block's channels, a channel a thread, all tokens' operands in flight together; then every warp forms both gates'
// sums of SO / 8 outputs for all tokens: lanes share the channels of a weight row (asked for before the wait for the
// projection while it fits: no kernel writes it), and a butterfly leaves every lane one sum.
constexpr int SO = 32, ST = 4, STEP_THREADS = 256, OW = SO / 8;
static_assert(OW * 2 * ST == 32, "one sum a lane");

template <typename TW> struct Unit { static constexpr int N = 4; };
template <> struct Unit<__nv_bfloat16> { static constexpr int N = 8; };
__device__ __forceinline__ void unpack(const uint4 v, float* f, float) {
  f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y); f[2] = __uint_as_float(v.z); f[3] = __uint_as_float(v.w);
}
__device__ __forceinline__ void unpack(const uint4 v, float* f, __nv_bfloat16) {
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(w[i] << 16);
    f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}

template <typename TW, typename TO>
__global__ void __launch_bounds__(STEP_THREADS, 2)
rglru_step_kernel(const float* __restrict__ proj, int n_partials, long long partial_stride, const float* __restrict__ bias,
                  const float* __restrict__ conv_w, const float* __restrict__ conv_b, int taps, const TW* __restrict__ wr,
                  const float* __restrict__ br, const TW* __restrict__ wi, const float* __restrict__ bi,
                  const float* __restrict__ rate, const int* __restrict__ pos, const int* __restrict__ slot,
                  float* __restrict__ state, long long state_stride, TO* __restrict__ out, int T, int W, int n, int vec) {
  extern __shared__ __align__(16) float sm[];  // us [ST][n], then xs [ST][SO], then z [ST][SO][2]
  __shared__ long long home_s[ST];
  __shared__ long long ring_s[64][ST];         // where the input d positions back lies (a tap that looks before the start: -1)
  float* us = sm;
  float* xs = us + (size_t)ST * n;
  float* z = xs + ST * SO;
  constexpr int VN = Unit<TW>::N;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int slices = (n + SO - 1) / SO;
  const int blk = blockIdx.x / slices, o0 = (blockIdx.x % slices) * SO, t0 = blockIdx.y * ST;
  const int nt = min(ST, T - t0);
  // the first (for short rows: the only) units of this warp's weight rows
  uint4 first[OW][2];
#pragma unroll
  for (int j = 0; j < OW; ++j)
#pragma unroll
    for (int g = 0; g < 2; ++g) {
      const int o = o0 + warp * OW + j;
      first[j][g] = make_uint4(0u, 0u, 0u, 0u);
      if (vec && o < n && lane * VN < n)
        first[j][g] = *reinterpret_cast<const uint4*>((g ? wi : wr) + ((size_t)blk * n + o) * n + lane * VN);
    }
  if (tid < ST) {
    const int t = t0 + min(tid, nt - 1);
    home_s[tid] = (long long)slot[t] * state_stride;
  }
  for (int i = tid; i < taps * ST; i += STEP_THREADS) {
    const int d = i / ST, t = t0 + min(i % ST, nt - 1), p = pos[t];
    ring_s[d][i % ST] = p >= d ? (long long)slot[t] * state_stride + W + (long long)((p - d) % taps) * W : -1;
  }
  __syncthreads();
  pdl_launch();
  pdl_wait();
  for (int k = tid; k < n; k += STEP_THREADS) {
    const int c = blk * n + k;
    const float* src = proj + (size_t)t0 * 2 * W + W + c;
    float x[ST], u[ST];
#pragma unroll
    for (int t = 0; t < ST; ++t) { x[t] = 0.f; u[t] = conv_b[c]; }
#pragma unroll 4
    for (int q = 0; q < n_partials; ++q)
#pragma unroll
      for (int t = 0; t < ST; ++t)
        if (t < nt) x[t] += src[(size_t)q * partial_stride + (size_t)t * 2 * W];
#pragma unroll 3
    for (int d = taps - 1; d >= 1; --d) {
      const float w = conv_w[(size_t)c * taps + taps - 1 - d];
#pragma unroll
      for (int t = 0; t < ST; ++t)
        if (t < nt && ring_s[d][t] >= 0) u[t] = fmaf(w, state[ring_s[d][t] + c], u[t]);
    }
    const float w = conv_w[(size_t)c * taps + taps - 1], bx = bias[W + c];
#pragma unroll
    for (int t = 0; t < ST; ++t) {
      x[t] += bx;
      us[t * n + k] = t < nt ? fmaf(w, x[t], u[t]) : 0.f;
      if (k >= o0 && k < o0 + SO) xs[t * SO + k - o0] = x[t];
    }
  }
  __syncthreads();
  float acc[OW * 2 * ST];                     // index (j * 2 + gate) * ST + token
#pragma unroll
  for (int i = 0; i < OW * 2 * ST; ++i) acc[i] = 0.f;
  if (vec) {
    for (int k = lane * VN; k < n; k += 32 * VN) {
      float w[OW][2][VN];
#pragma unroll
      for (int j = 0; j < OW; ++j)
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          const int o = min(o0 + warp * OW + j, n - 1);
          const uint4 v = k == lane * VN ? first[j][g]
                                         : *reinterpret_cast<const uint4*>((g ? wi : wr) + ((size_t)blk * n + o) * n + k);
          unpack(v, w[j][g], TW());
        }
#pragma unroll
      for (int t = 0; t < ST; ++t)
#pragma unroll
        for (int v = 0; v < VN; v += 4) {
          const float4 x = *reinterpret_cast<const float4*>(us + t * n + k + v);
#pragma unroll
          for (int j = 0; j < OW; ++j)
#pragma unroll
            for (int g = 0; g < 2; ++g) {
              float& s = acc[(j * 2 + g) * ST + t];
              s = fmaf(w[j][g][v], x.x, s); s = fmaf(w[j][g][v + 1], x.y, s);
              s = fmaf(w[j][g][v + 2], x.z, s); s = fmaf(w[j][g][v + 3], x.w, s);
            }
        }
    }
  } else {
    for (int k = lane; k < n; k += 32)
#pragma unroll
      for (int j = 0; j < OW; ++j)
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          const int o = min(o0 + warp * OW + j, n - 1);
          const float w = to_f32((g ? wi : wr)[((size_t)blk * n + o) * n + k]);
#pragma unroll
          for (int t = 0; t < ST; ++t) acc[(j * 2 + g) * ST + t] = fmaf(w, us[t * n + k], acc[(j * 2 + g) * ST + t]);
        }
  }
  // 32 sums over 32 lanes: each exchange halves how many a lane holds; lane l ends with the sum of index l
#pragma unroll
  for (int m = 16; m >= 1; m >>= 1) {
    const bool up = lane & m;
#pragma unroll
    for (int i = 0; i < m; ++i) {
      const float give = up ? acc[i] : acc[i + m], keep = up ? acc[i + m] : acc[i];
      acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, m);
    }
  }
  z[((lane % ST) * SO + warp * OW + lane / (2 * ST)) * 2 + (lane / ST) % 2] = acc[0];
  __syncthreads();
  for (int i = tid; i < nt * SO; i += STEP_THREADS) {
    const int tt = i / SO, j = i % SO, o = o0 + j, t = t0 + tt;
    if (o >= n) continue;
    const int c = blk * n + o;
    const float* src = proj + (size_t)t * 2 * W + c;
    float y = bias[c];
#pragma unroll 4
    for (int q = 0; q < n_partials; ++q) y += src[(size_t)q * partial_stride];
    float a, b;
    unit(z[i * 2] + br[c], z[i * 2 + 1] + bi[c], rate[c], us[tt * n + o], a, b);
    float* home = state + home_s[tt];
    const float S = fmaf(a, home[c], b);
    home[c] = S;
    state[ring_s[0][tt] + c] = xs[i];
    out[(size_t)t * W + c] = from_f32<TO>(S * gelu_tanhf_(y));
  }
}

}  // namespace

// u [T, W] float32; wr, wi [B, n, n] (out, in) with W = B n; br, bi, rate [W] float32; a, b [T, W] float32.
extern "C" int flint_rglru_gates(const float* u, const void* wr, const float* br, const void* wi, const float* bi,
                                 int w_dtype, const float* rate, float* a, float* b, int T, int W, int blocks, int tensor,
                                 cudaStream_t stream) {
  if (T <= 0) return 0;
  if (blocks < 1 || W < 1 || W % blocks) return fail("rglru_gates: %d channels do not form %d equal blocks", W, blocks);
  if (blocks > 65535) return fail("rglru_gates: too many blocks (%d)", blocks);
  const int n = W / blocks;
  if (tensor) {
    if (w_dtype != FLINT_BF16 || n % 8 || ((uintptr_t)wr & 15) || ((uintptr_t)wi & 15) || ((uintptr_t)u & 15) ||
        ((uintptr_t)a & 7) || ((uintptr_t)b & 7))
      return fail("rglru_gates: the tensor-core form takes bfloat16 blocks of a multiple of 8 channels, 16-byte aligned");
    launch_pdl(gates_mma_kernel, dim3((T + MM - 1) / MM, (n + MN - 1) / MN, blocks), dim3(128), 0, stream, u,
               (const __nv_bfloat16*)wr, br, (const __nv_bfloat16*)wi, bi, rate, a, b, T, W, n);
    return check_launch("rglru_gates (tensor cores)");
  }
  FLINT_DISPATCH_DTYPE(w_dtype, TW,
      launch_pdl(gates_simt_kernel<TW>, dim3((T + GM - 1) / GM, (n + GN - 1) / GN, blocks), dim3(256), 0, stream, u,
                 (const TW*)wr, br, (const TW*)wi, bi, rate, a, b, T, W, n));
  return check_launch("rglru_gates");
}

// Rows a chunk of the scan holds: the caller sizes `totals` by it.
extern "C" int flint_rglru_chunk() { return CHUNK; }

// a, b [T, W]; y [T, W] float32 with a row stride; request e owns rows seq_start[e] .. seq_start[e + 1] - 1 (null: row e
// alone); longest: the most rows any request owns; state: the first W floats of each slot's row; totals
// [n_seq, ceil(longest / chunk) + 1, 2, W] floats when longest exceeds a chunk, else null; out [T, W].
extern "C" int flint_rglru_scan(const float* a, const float* b, const float* y, long long y_stride, const int* slot,
                                const int* seq_start, int n_seq, int longest, float* state, long long state_stride,
                                float* totals, void* out, int out_dtype, int W, cudaStream_t stream) {
  if (n_seq <= 0 || longest <= 0 || W <= 0) return 0;
  const int chunks = (longest + CHUNK - 1) / CHUNK;
  if (chunks > 1 && !totals) return fail("rglru_scan: rows beyond one chunk need the totals' memory");
  if (n_seq > 65535 || chunks > 65535) return fail("rglru_scan: too many requests or rows");
  const int threads = W >= 128 ? 128 : 64;
  const dim3 grid((W + threads - 1) / threads, chunks, n_seq);
  if (chunks > 1)
    launch_pdl(rglru_totals_kernel, grid, dim3(threads), 0, stream, a, b, slot, seq_start, (const float*)state, state_stride,
               totals, chunks, W);
  FLINT_DISPATCH_DTYPE(out_dtype, TO,
      launch_pdl(rglru_walk_kernel<TO>, grid, dim3(threads), 0, stream, a, b, y, y_stride, slot, seq_start, state,
                 state_stride, (const float*)(chunks > 1 ? totals : nullptr), chunks, (TO*)out, W));
  return check_launch("rglru_scan");
}

// proj [S, T, 2 W] float32 partial sums of the two branches' projection ([y | x], bias [2 W] apart); conv_w [W, taps],
// conv_b [W]; state rows [S (W) | taps rows of W inputs]; one row per request; out [T, W].
extern "C" int flint_rglru_step(const float* proj, int n_partials, long long partial_stride, const float* bias,
                                const float* conv_w, const float* conv_b, int taps, const void* wr, const float* br,
                                const void* wi, const float* bi, int w_dtype, const float* rate, const int* pos,
                                const int* slot, float* state, long long state_stride, void* out, int out_dtype, int T,
                                int W, int blocks, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (blocks < 1 || W < 1 || W % blocks) return fail("rglru_step: %d channels do not form %d equal blocks", W, blocks);
  if (taps < 1 || taps > 64) return fail("rglru_step: %d taps are not supported (1 to 64)", taps);
  if (n_partials < 1) return fail("rglru_step: needs at least one partial");
  const int n = W / blocks, slices = (n + SO - 1) / SO;
  const size_t smem = ((size_t)ST * n + 3 * ST * SO) * sizeof(float);
  if (smem > 200 * 1024) return fail("rglru_step: blocks of %d channels are not supported", n);
  if ((T + ST - 1) / ST > 65535) return fail("rglru_step: too many rows");
  const int vec = n % (w_dtype == FLINT_BF16 ? 8 : 4) == 0 && !(((uintptr_t)wr | (uintptr_t)wi) & 15);
  const dim3 grid((unsigned)(blocks * slices), (unsigned)((T + ST - 1) / ST));
  FLINT_DISPATCH_DTYPE(w_dtype, TW, FLINT_DISPATCH_DTYPE(out_dtype, TO, {
    if (smem > 48 * 1024)
      cudaFuncSetAttribute(rglru_step_kernel<TW, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    launch_pdl(rglru_step_kernel<TW, TO>, grid, dim3(STEP_THREADS), smem, stream, proj, n_partials, partial_stride, bias,
               conv_w, conv_b, taps, (const TW*)wr, br, (const TW*)wi, bi, rate, pos, slot, state, state_stride, (TO*)out, T,
               W, n, vec);
  }));
  return check_launch("rglru_step");
}

extern "C" const char* flint_rglru_last_error() { return g_error; }
