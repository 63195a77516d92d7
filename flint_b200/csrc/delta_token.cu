// The gated delta rule for a batch of single tokens, from the projection to the normed and gated heads, in one launch (the
// form with one decay a head and a full gate):
//
//   q, k, v   = silu(causal convolution of the projected columns);   q, k unit vectors per head, q times D^(-1/2)
//   beta      = sigmoid(b);   g = exp(-exp(A_log) softplus(a + dt_bias))
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   out       = o / rms(o) * w * act(gate)
//
// One block per (request, head).  The head's matrix S [D, V] lies in registers: a warp takes rows d = warp, warp + 16, ..., a
// lane a few neighbouring columns of each, so every row is read and written in whole runs; the dot products over the rows
// meet through shared memory, twice a token.  S and the convolution's earlier inputs are last written by an earlier step, which
// has ended, so the matrix is on its way before the wait for the projection (two launches on the same state must not follow
// each other in a stream without another kernel between them).  The projection arrives as partial
// sums, the convolution's inputs of the past lie in a ring of `taps` rows of the request's state (the input of position p in
// row p mod taps): the row a token writes is none that its own convolution reads, so the heads that share a key head need no
// order.  Everything is float32.  The reference runs its delta rule token by token on recurrent state per sequence as well
// (crates/thuban_architectures/src/qwen35/state.rs:5-55).
#include <math.h>
#include <stdarg.h>
#include "common.cuh"

using namespace flint;

namespace {

constexpr int NW = 16;                   // warps a block

struct TokenArgs {
  const float* proj; int n_partials; long long partial_stride; int width;      // columns q | k | v | b | a | gate
  const float* conv_w; int taps;
  const float* dt_bias; const float* a_log; const float* norm_w;
  const int* pos; const int* slot;
  float* state; long long state_stride;                                        // rows: S of every head, then the ring
  float unit_eps, eps; int gate_silu;
  int H, G, D, V;
};

__device__ __forceinline__ float sigmoidf_(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float siluf_(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplusf_(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

template <int CPL> struct Cols;
template <> struct Cols<1> {
  static __device__ __forceinline__ void load(const float* p, float* v) { v[0] = *p; }
  static __device__ __forceinline__ void store(float* p, const float* v) { *p = v[0]; }
};
template <> struct Cols<2> {
  static __device__ __forceinline__ void load(const float* p, float* v) {
    const float2 x = *reinterpret_cast<const float2*>(p);
    v[0] = x.x; v[1] = x.y;
  }
  static __device__ __forceinline__ void store(float* p, const float* v) { *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]); }
};
template <> struct Cols<4> {
  static __device__ __forceinline__ void load(const float* p, float* v) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};

// RW: rows of S a warp holds (D <= 16 RW); CPL: columns a lane holds (32 CPL columns at a time); BLOCKS: blocks a multiprocessor
// (one with all the registers it wants, or, where there are more blocks than multiprocessors, two)
template <int RW, int CPL, int BLOCKS, typename TO>
__global__ void __launch_bounds__(NW * 32, BLOCKS)
delta_token_kernel(const __grid_constant__ TokenArgs a, TO* __restrict__ out) {
  extern __shared__ __align__(16) float sm[];          // sums of the warps [NW][32 CPL], then q [D], k [D], v [V], gate [V], o [V]
  __shared__ float scalars[2], red[32];
  const int h = blockIdx.x, e = blockIdx.y, D = a.D, V = a.V, kh = h / (a.H / a.G);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  constexpr int COLS = 32 * CPL;
  float *part = sm, *q_s = part + NW * COLS, *k_s = q_s + D, *v_s = k_s + D, *g_s = v_s + V, *o_s = g_s + V;
  const int p = a.pos[e];
  float* mine = a.state + (size_t)a.slot[e] * a.state_stride;
  float* S_g = mine + (size_t)h * D * V;
  float S[RW][CPL];
  auto load_state = [&](int c) {
#pragma unroll
    for (int i = 0; i < RW; ++i) {
      const int d = warp + NW * i;
#pragma unroll
      for (int j = 0; j < CPL; ++j) S[i][j] = 0.f;
      if (d < D && c < V) Cols<CPL>::load(S_g + (size_t)d * V + c, S[i]);
    }
  };
  load_state(lane * CPL);
  pdl_launch();
  pdl_wait();
  // ---- the head's operands
  const float* row = a.proj + (size_t)e * a.width;
  auto projected = [&](int c) {
    float x = 0.f;
    for (int z = 0; z < a.n_partials; ++z) x += row[(size_t)z * a.partial_stride + c];
    return x;
  };
  const int GD = a.G * D, HV = a.H * V, C = 2 * GD + HV;
  float* ring = mine + (size_t)a.H * D * V;
  const bool keeps_qk = h % (a.H / a.G) == 0;                // one of the heads that share q and k stores their inputs
  for (int i = tid; i < 2 * D + V; i += NW * 32) {
    const int c = i < D ? kh * D + i : i < 2 * D ? GD + kh * D + (i - D) : 2 * GD + h * V + (i - 2 * D);
    const float x = projected(c);
    const float* w = a.conv_w + (size_t)c * a.taps;
    float acc = 0.f;
    for (int d = a.taps - 1; d >= 1; --d)                    // oldest first, as over prompts
      if (p >= d) acc = fmaf(w[a.taps - 1 - d], ring[(size_t)((p - d) % a.taps) * C + c], acc);
    acc = fmaf(w[a.taps - 1], x, acc);
    q_s[i] = siluf_(acc);                                    // q | k | v lie one behind the other
    if (a.taps > 1 && (i >= 2 * D || keeps_qk)) ring[(size_t)(p % a.taps) * C + c] = x;
  }
  for (int i = tid; i < V; i += NW * 32) g_s[i] = projected(C + 2 * a.H + h * V + i);
  if (tid == 0) scalars[0] = sigmoidf_(projected(C + h));
  if (tid == 32) scalars[1] = expf(-expf(a.a_log[h]) * softplusf_(projected(C + a.H + h) + a.dt_bias[h]));
  __syncthreads();
  if (warp < 2) {                                            // unit vectors
    float* x = warp == 0 ? q_s : k_s;
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) ss = fmaf(x[d], x[d], ss);
    const float inv = (1.0f / sqrtf(warp_sum(ss) + a.unit_eps)) * (warp == 0 ? rsqrtf((float)D) : 1.0f);
    for (int d = lane; d < D; d += 32) x[d] *= inv;
  }
  __syncthreads();
  const float beta = scalars[0], decay = scalars[1];
  auto key = [&](int i) { return warp + NW * i < D ? k_s[warp + NW * i] : 0.f; };        // of the warp's i-th row
  auto query = [&](int i) { return warp + NW * i < D ? q_s[warp + NW * i] : 0.f; };
  // ---- the recurrence, a run of columns at a time
  float sq = 0.f;
  for (int c0 = 0; c0 < V; c0 += COLS) {
    const int c = c0 + lane * CPL;
    if (c0 > 0) load_state(c);
    float acc[CPL];
#pragma unroll
    for (int j = 0; j < CPL; ++j) acc[j] = 0.f;
#pragma unroll
    for (int i = 0; i < RW; ++i) {
      const float kd = key(i);
#pragma unroll
      for (int j = 0; j < CPL; ++j) {
        S[i][j] *= decay;
        acc[j] = fmaf(S[i][j], kd, acc[j]);
      }
    }
    Cols<CPL>::store(part + warp * COLS + lane * CPL, acc);
    __syncthreads();
    float u[CPL];
#pragma unroll
    for (int j = 0; j < CPL; ++j) u[j] = 0.f;
    for (int w = 0; w < NW; ++w) {                           // the same order in every warp
      float t[CPL];
      Cols<CPL>::load(part + w * COLS + lane * CPL, t);
#pragma unroll
      for (int j = 0; j < CPL; ++j) u[j] += t[j];
    }
#pragma unroll
    for (int j = 0; j < CPL; ++j) {
      u[j] = c + j < V ? beta * (v_s[c + j] - u[j]) : 0.f;
      acc[j] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < RW; ++i) {
      const float kd = key(i), qd = query(i);
#pragma unroll
      for (int j = 0; j < CPL; ++j) {
        S[i][j] = fmaf(kd, u[j], S[i][j]);
        acc[j] = fmaf(S[i][j], qd, acc[j]);
      }
      const int d = warp + NW * i;
      if (d < D && c < V) Cols<CPL>::store(S_g + (size_t)d * V + c, S[i]);
    }
    __syncthreads();                                         // the sums of S^T k have been read
    Cols<CPL>::store(part + warp * COLS + lane * CPL, acc);
    __syncthreads();
    if (tid < COLS && c0 + tid < V) {
      float o = 0.f;
      for (int w = 0; w < NW; ++w) o += part[w * COLS + tid];
      o_s[c0 + tid] = o;
      sq = fmaf(o, o, sq);
    }
    __syncthreads();
  }
  // ---- norm and gate
  const float inv = 1.0f / sqrtf(block_sum(sq, red) / (float)V + a.eps);
  for (int i = tid; i < V; i += NW * 32) {
    const float gt = a.gate_silu ? siluf_(g_s[i]) : sigmoidf_(g_s[i]);
    out[(size_t)e * HV + (size_t)h * V + i] = from_f32<TO>(o_s[i] * inv * a.norm_w[i] * gt);
  }
}

template <int RW, int CPL, int BLOCKS, typename TO>
void launch_form(const TokenArgs& a, int n, TO* out, size_t smem, cudaStream_t stream) {
  static bool sized = false;             // per instantiation
  if (smem > 48 * 1024 && !sized) {
    cudaFuncSetAttribute(delta_token_kernel<RW, CPL, BLOCKS, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    sized = true;
  }
  launch_pdl(delta_token_kernel<RW, CPL, BLOCKS, TO>, dim3((unsigned)a.H, (unsigned)n), dim3(NW * 32), smem, stream, a, out);
}

template <int RW, int CPL>
int launch_token(const TokenArgs& a, int n, void* out, int out_dtype, size_t smem, cudaStream_t stream) {
  constexpr int MORE = RW * CPL <= 32 ? 2 : 1;
  static int sms = 0;
  if (!sms) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  }
  const bool many = (long long)a.H * n > sms;
  FLINT_DISPATCH_DTYPE(out_dtype, TO, {
    if (many) launch_form<RW, CPL, MORE, TO>(a, n, (TO*)out, smem, stream);
    else launch_form<RW, CPL, 1, TO>(a, n, (TO*)out, smem, stream);
  });
  return check_launch("delta_token");
}
}  // namespace

// proj [n_partials, n, width] float32 (stride partial_stride): columns q (G D) | k (G D) | v (H V) | b (H) | a (H) | gate (H V);
// conv_w [2 G D + H V, taps]; dt_bias, a_log [H]; norm_w [V]; row i is request slot[i]'s token at position pos[i]; state rows
// (stride state_stride floats) hold S [H, D, V] and, with taps > 1, a ring of `taps` rows of the 2 G D + H V convolved inputs, and
// are brought up to date; out [n, H V] in out_dtype.
extern "C" int flint_delta_token(const float* proj, int n_partials, long long partial_stride, int width, const float* conv_w,
                                 int taps, const float* dt_bias, const float* a_log, const float* norm_w, const int* pos,
                                 const int* slot, float* state, long long state_stride, float unit_eps, float eps, int gate_silu,
                                 void* out, int out_dtype, int n, int H, int G, int D, int V, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (D < 1 || D > 256 || V < 1) return fail("delta_token: %d key dims per head are not supported (1 to 256)", D);
  if (G <= 0 || H % G) return fail("delta_token: %d heads do not divide into %d key heads", H, G);
  if (n_partials < 1 || width != 2 * G * D + 2 * H * V + 2 * H) return fail("delta_token: the projection's width does not match the sizes");
  if (taps < 1 || taps > 64) return fail("delta_token: %d taps are not supported (1 to 64)", taps);
  if (n > 65535) return fail("delta_token: too many requests");
  TokenArgs a = {};
  a.proj = proj; a.n_partials = n_partials; a.partial_stride = partial_stride; a.width = width;
  a.conv_w = conv_w; a.taps = taps; a.dt_bias = dt_bias; a.a_log = a_log; a.norm_w = norm_w; a.pos = pos; a.slot = slot;
  a.state = state; a.state_stride = state_stride; a.unit_eps = unit_eps; a.eps = eps; a.gate_silu = gate_silu;
  a.H = H; a.G = G; a.D = D; a.V = V;
  // a lane's columns in one access: the rows of S must start on its boundary
  auto lined = [&](int c) { return V % c == 0 && state_stride % c == 0 && ((uintptr_t)state & (4 * c - 1)) == 0; };
  const int cpl = V > 64 && lined(4) ? 4 : V > 32 && lined(2) ? 2 : 1;
  const int rw = D <= 32 ? 2 : D <= 64 ? 4 : D <= 128 ? 8 : 16;
  const size_t smem = ((size_t)2 * D + 3 * V + NW * 32 * cpl) * sizeof(float);
  if (smem > 200 * 1024) return fail("delta_token: heads of %d and %d dims are not supported", D, V);
#define GO(RW) (cpl == 4 ? launch_token<RW, 4>(a, n, out, out_dtype, smem, stream) \
                : cpl == 2 ? launch_token<RW, 2>(a, n, out, out_dtype, smem, stream) : launch_token<RW, 1>(a, n, out, out_dtype, smem, stream))
  if (rw == 2) return GO(2);
  if (rw == 4) return GO(4);
  if (rw == 8) return GO(8);
  return GO(16);
#undef GO
}

extern "C" const char* flint_delta_token_last_error() { return g_error; }
