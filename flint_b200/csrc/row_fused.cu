// The row kernel of the residual stream: apply what earlier kernels left pending, normalise,
// and (optionally) route -- one block per row, or for a handful of rows a cluster of blocks per row, the row
// held in registers.
//
//   x[row] += sum_z partials[z][row] + bias          (a product whose K range was split)
//   x[row] += g0 * y[r0] + g1 * y[r1]                 (the two selected experts' outputs)
//   y = LayerNorm(x[row]) or RMSNorm(x[row])          float32 statistics, two passes over registers
//   out_f32 / out_bf16 <- y
//
// With several streams a row [S, H] is kept instead of x[row] [H]: with r what is pending (the two additions above),
//
//   x_t[row] <- sum_s mix[s, t] x_s[row] + out[t] r       (all t from the old streams; only with something pending)
//   y = norm(sum_s gather[s] x_s[row])
//
//   logits_e = <y, Wr[e]>, sparsemixer top-2          (float32; same selection as moe.cu)
//
// Fusing these saves, per layer of a decode step, the kernels that would only add to the
// residual stream and one pass over it.  Widths that are not a multiple of 4 or exceed 16384
// are refused; the caller then uses the separate kernels.
// Reference counterparts: crates/thuban_kernel/wgsl/norm.wgsl (mode 3), add.wgsl, merge_gemm.wgsl.
#include <math.h>
#include <stdarg.h>
#include "common.cuh"
#include "router_select.cuh"

using namespace flint;

namespace {
constexpr int MAX_VPT = 4;
constexpr int MAX_E = 256;
constexpr int FUSED_STREAMS = 4;         // streams the row kernel takes (their columns are held in registers)
constexpr int MAX_STREAMS = 16;          // streams the update kernel takes

struct RowArgs {
  float* x;
  const int* row_index;
  const float* partials; int n_partials; long long partial_stride; const float* add_bias;
  const float* comb_y; const int* comb_row_of; const float* comb_gates; int comb_top;
  const float* gamma; const float* beta; float eps; int mode;
  float* out_f32; __nv_bfloat16* out_bf16;
  const void* wr; int E; float jitter_eps; int* expert_ids; float* gates;
  int top, n_groups, keep; float out_scale;      // top > 0: the softmax router limited to groups instead of sparsemixer
  int rule, extra; float* aux;  // rule 1: the sigmoid router (scores into gates, the last `extra` rows of wr are gates: aux)
  const float* correction; int normalize;   // rule 2: the sigmoid router limited to groups (select_corrected_by_warp); rule 3: the same over a softmax
  float* router_logits;        // optional [rows, E]: the logits the selection was made from (for tests)
  int n_streams;               // > 0: x is [rows, n_streams, H]; the mixing weights of what is pending, of the norm's input
  const float* mix; const float* spread; const float* gather;
  int store;                   // streams: whether the new streams are written back
  int H;
};

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void add4(float4& a, const float4 b) { a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w; }
__device__ __forceinline__ void fma4(float4& a, float g, const float4 b) {
  a.x = fmaf(g, b.x, a.x); a.y = fmaf(g, b.y, a.y); a.z = fmaf(g, b.z, a.z); a.w = fmaf(g, b.w, a.w);
}

__device__ __forceinline__ void load_w8(const float* p, float* f) {
  const float4 a = ld4(p), b = ld4(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void load_w8(const __nv_bfloat16* p, float* f) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(w[i] << 16);
    f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}

// The mixing weights of a kernel's streams, staged in shared memory (they are weights: no kernel writes them).
template <int ST>
struct StreamWeights { float mix[ST > 0 ? ST * ST : 1], spread[ST > 0 ? ST : 1], gather[ST > 0 ? ST : 1]; };

template <int ST>
__device__ __forceinline__ void load_stream_weights(StreamWeights<ST>& w, const RowArgs& a) {
  for (int i = threadIdx.x; i < a.n_streams * a.n_streams; i += blockDim.x) w.mix[i] = a.mix ? a.mix[i] : 0.f;
  for (int i = threadIdx.x; i < a.n_streams; i += blockDim.x) {
    w.spread[i] = a.spread ? a.spread[i] : 0.f;
    w.gather[i] = a.gather ? a.gather[i] : 0.f;
  }
}

// Four neighbouring columns of one row's streams: bring them up to date with what is pending (r), store them, and
// return the norm's input.  xr: the row's first stream, at the columns.
template <int ST>
__device__ __forceinline__ float4 stream_columns(float* xr, const float4 r, const StreamWeights<ST>& w, const RowArgs& a,
                                                 bool pending) {
  float4 x[ST > 0 ? ST : 1];
  const int n = a.n_streams;
#pragma unroll
  for (int s = 0; s < ST; ++s) x[s] = s < n ? ld4(xr + (size_t)s * a.H) : make_float4(0.f, 0.f, 0.f, 0.f);
  float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int t = 0; t < ST; ++t) {
    if (t >= n) break;
    float4 v = x[t];
    if (pending) {
      v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < ST; ++s)
        if (s < n) fma4(v, w.mix[s * n + t], x[s]);
      fma4(v, w.spread[t], r);
      if (a.store) *reinterpret_cast<float4*>(xr + (size_t)t * a.H) = v;
    }
    fma4(u, w.gather[t], v);
  }
  return u;
}

// sparsemixer top-2 of one row (float32; same selection as moe.cu).  Up to 32 experts sit one per lane of a
// warp (arg-max and the masked sums by shuffle).
__device__ __forceinline__ void select_two_by_lanes(float sv, int lane, int E, float jitter_eps, int* ids, float* gates) {
  int excluded = -1;
  for (int round = 0; round < 2; ++round) {
    // arg-max over lanes, lowest index on ties
    float m = (lane < E && lane != excluded) ? sv : -INFINITY;
    int im = lane;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float om = __shfl_xor_sync(0xffffffffu, m, o);
      const int oi = __shfl_xor_sync(0xffffffffu, im, o);
      if (om > m || (om == m && oi < im)) { m = om; im = oi; }
    }
    float term = 0.f;
    if (lane < E && lane != excluded) {
      const float factor = fmaxf(fabsf(sv), m);
      if (!(((m - sv) / factor) > 2.0f * jitter_eps)) term = expf(sv - m);
    }
    // the sum in lane order, so that it does not depend on the shuffle tree
    float denom = 0.f;
    for (int e = 0; e < E; ++e) denom += __shfl_sync(0xffffffffu, term, e);
    if (lane == 0) {
      ids[round] = im;
      gates[round] = 1.0f / denom;
    }
    excluded = im;
  }
}
// any number of experts, by one thread
__device__ __forceinline__ void select_two_serial(const float* s, int E, float jitter_eps, int* ids, float* gates) {
  int excluded = -1;
  for (int round = 0; round < 2; ++round) {
    float m = -INFINITY;
    int im = 0;
    for (int e = 0; e < E; ++e)
      if (e != excluded && s[e] > m) { m = s[e]; im = e; }
    float denom = 0.f;
    for (int e = 0; e < E; ++e) {
      if (e == excluded) continue;
      const float factor = fmaxf(fabsf(s[e]), m);
      if (!(((m - s[e]) / factor) > 2.0f * jitter_eps)) denom += expf(s[e] - m);
    }
    ids[round] = im;
    gates[round] = 1.0f / denom;
    excluded = im;
  }
}

// The router of one row, by its block: smem holds the H float32 numbers of the row (written by any of the block's threads),
// then room for the partial logits.
template <typename TW>
__device__ __forceinline__ void route_by_block(const RowArgs& a, float* smem) {
  const int H = a.H;
  // ---- router: a job is (group of 4 experts, strided share of the row); a warp keeps 4 sums, so that
  // every value read from shared memory feeds 4 multiply-adds; partial sums meet in shared memory
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const int E = a.E;
  constexpr int EG = 4;
  const int groups = (E + EG - 1) / EG;
  const int k = n_warps >= groups ? n_warps / groups : 1;   // warps per expert group
  float* part = smem + H;                                    // [E][k]
  const TW* wr = (const TW*)a.wr;
  const bool vec = (H & 7) == 0;
  for (int job = warp; job < groups * k; job += n_warps) {
    const int e0 = (job / k) * EG, sl = job % k;
    float acc[EG];
#pragma unroll
    for (int j = 0; j < EG; ++j) acc[j] = 0.f;
    if (vec) {
#pragma unroll 2
      for (int d = (sl * 32 + lane) * 8; d < H; d += k * 256) {
        float wv[EG][8];
#pragma unroll
        for (int j = 0; j < EG; ++j) {
          if (e0 + j < E) {
            load_w8(wr + (size_t)(e0 + j) * H + d, wv[j]);
          } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) wv[j][i] = 0.f;
          }
        }
        const float4 x0 = ld4(smem + d), x1 = ld4(smem + d + 4);
        const float xv[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
        for (int j = 0; j < EG; ++j)
#pragma unroll
          for (int i = 0; i < 8; ++i) acc[j] = fmaf(xv[i], wv[j][i], acc[j]);
      }
    } else {
      for (int d = sl * 32 + lane; d < H; d += k * 32) {
        const float xv = smem[d];
#pragma unroll
        for (int j = 0; j < EG; ++j)
          acc[j] = fmaf(xv, e0 + j < E ? to_f32(wr[(size_t)(e0 + j) * H + d]) : 0.f, acc[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < EG; ++j) {
      const float t = warp_sum(acc[j]);
      if (lane == 0 && e0 + j < E) part[(e0 + j) * k + sl] = t;
    }
  }
  __syncthreads();
  // selection by the first warp.  Up to 32 experts sit one per lane (argmax and the masked sums by
  // shuffle); more experts are handled by lane 0 alone.
  if (warp != 0) return;
  const int r = blockIdx.x;
  if (a.top > 0) {                                         // softmax router limited to groups: the warp selects
    float* s = smem;                                       // the row is no longer needed
    for (int e = lane; e < E; e += 32) {
      float t = 0.f;
      for (int i = 0; i < k; ++i) t += part[e * k + i];    // fixed order
      s[e] = t;
      if (a.router_logits) a.router_logits[(size_t)r * E + e] = t;
    }
    __syncwarp();
    if (a.rule >= 2)
      select_corrected_by_warp(s, s + E, a.correction, a.rule == 3, lane, E, a.top, a.n_groups, a.keep, a.normalize, a.out_scale,
                                     a.expert_ids + (size_t)a.top * r, a.gates + (size_t)a.top * r);
    else if (a.rule == 1)
      select_sigmoid_by_warp(s, lane, E - a.extra, a.extra, a.top, a.expert_ids + (size_t)a.top * r,
                             a.gates + (size_t)a.top * r, a.aux + (size_t)(a.top + a.extra) * r);
    else
      select_topk_by_warp(s, lane, E, a.top, a.n_groups, a.keep, a.out_scale, a.expert_ids + (size_t)a.top * r,
                          a.gates + (size_t)a.top * r);
    return;
  }
  if (E <= 32) {
    float sv = -INFINITY;
    if (lane < E) {
      sv = 0.f;
      for (int i = 0; i < k; ++i) sv += part[lane * k + i];    // fixed order
      if (a.router_logits) a.router_logits[(size_t)r * E + lane] = sv;
    }
    select_two_by_lanes(sv, lane, E, a.jitter_eps, a.expert_ids + 2 * r, a.gates + 2 * r);
    return;
  }
  if (lane != 0) return;
  float* s = smem;                                         // the row is no longer needed
  for (int e = 0; e < E; ++e) {
    float t = 0.f;
    for (int i = 0; i < k; ++i) t += part[e * k + i];    // fixed order
    s[e] = t;
    if (a.router_logits) a.router_logits[(size_t)r * E + e] = t;
  }
  select_two_serial(s, E, a.jitter_eps, a.expert_ids + 2 * r, a.gates + 2 * r);
}

// One block per row; a thread holds VPT vectors of four values of its row.
// ST: 0 for a plain residual row, else the most streams this form takes.
template <int VPT, typename TW, int ST>
__global__ void __launch_bounds__(1024)
row_norm_kernel(const __grid_constant__ RowArgs a) {
  extern __shared__ float smem[];          // router only: H floats of the normalised row, then partial logits
  __shared__ float red[32];
  __shared__ StreamWeights<ST> hw;
  pdl_launch();
  if constexpr (ST > 0) {
    load_stream_weights<ST>(hw, a);
    __syncthreads();
  }
  pdl_wait();
  const int H = a.H, n4 = H >> 2;
  {
    const int r = blockIdx.x;
    const int src = a.row_index ? a.row_index[r] : r;
    float* xr = a.x + (size_t)src * (ST > 0 ? a.n_streams : 1) * H;
    float4 v[VPT];
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      v[i] = ST == 0 && c < n4 ? ld4(xr + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const bool pending = a.partials || a.comb_y;
    if (a.partials) {
      const float* pr = a.partials + (size_t)src * H;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < n4) {
          for (int z0 = 0; z0 < a.n_partials; z0 += 4) {      // four loads in flight, added in a fixed order
            float4 t[4];
#pragma unroll
            for (int u = 0; u < 4; ++u)
              t[u] = z0 + u < a.n_partials ? ld4(pr + (size_t)(z0 + u) * a.partial_stride + 4 * c)
                                           : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int u = 0; u < 4; ++u) add4(v[i], t[u]);
          }
        }
      }
      if (a.add_bias) {
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int c = threadIdx.x + i * blockDim.x;
          if (c < n4) add4(v[i], ld4(a.add_bias + 4 * c));
        }
      }
    }
    if (a.comb_y) {
      // the chosen experts' rows times their gates, summed in the order of the choices, then added: the order
      // of moe_combine
      float4 t[VPT];
#pragma unroll
      for (int i = 0; i < VPT; ++i) t[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int k = 0; k < a.comb_top; ++k) {
        const float g = a.comb_gates[(size_t)a.comb_top * src + k];
        const float* y = a.comb_y + (size_t)a.comb_row_of[(size_t)a.comb_top * src + k] * H;
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int c = threadIdx.x + i * blockDim.x;
          if (c < n4) fma4(t[i], g, ld4(y + 4 * c));
        }
      }
#pragma unroll
      for (int i = 0; i < VPT; ++i) add4(v[i], t[i]);
    }
    if constexpr (ST > 0) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < n4) v[i] = stream_columns<ST>(xr + 4 * c, v[i], hw, a, pending);
      }
    } else if (pending) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < n4) *reinterpret_cast<float4*>(xr + 4 * c) = v[i];
      }
    }
    if (!a.gamma) return;                     // only the additions were wanted
    // statistics
    float mean = 0.f;
    if (a.mode == 0) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < VPT; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);   // zeros beyond the row
      mean = block_sum(s, red) / (float)H;
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < n4) {
        const float d0 = v[i].x - mean, d1 = v[i].y - mean, d2 = v[i].z - mean, d3 = v[i].w - mean;
        ss += (d0 * d0 + d1 * d1) + (d2 * d2 + d3 * d3);
      }
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)H + a.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < n4) {
        const float4 g = ld4(a.gamma + 4 * c);
        float4 y = make_float4((v[i].x - mean) * inv * g.x, (v[i].y - mean) * inv * g.y,
                               (v[i].z - mean) * inv * g.z, (v[i].w - mean) * inv * g.w);
        if (a.beta) add4(y, ld4(a.beta + 4 * c));
        if (a.out_f32) *reinterpret_cast<float4*>(a.out_f32 + (size_t)r * H + 4 * c) = y;
        if (a.out_bf16) {
          const __nv_bfloat162 lo = __floats2bfloat162_rn(y.x, y.y), hi = __floats2bfloat162_rn(y.z, y.w);
          uint2 pk;
          pk.x = *reinterpret_cast<const uint32_t*>(&lo);
          pk.y = *reinterpret_cast<const uint32_t*>(&hi);
          *reinterpret_cast<uint2*>(a.out_bf16 + (size_t)r * H + 4 * c) = pk;
        }
        if (a.wr) *reinterpret_cast<float4*>(smem + 4 * c) = y;
      }
    }
  }
  if (!a.wr) return;
  route_by_block<TW>(a, smem);
}

// ---- few rows: a cluster of blocks per row
// With a handful of rows (a decode step) one block per row leaves the device empty and pulls the whole row,
// its pending partial sums and the router's weights through one SM.  Here the blocks of a cluster share a
// row: each takes a run of columns, the statistics and the router's partial sums meet through distributed
// shared memory (every block writes its share into the others' memory, one cluster barrier, then every block
// adds the shares in rank order, so all of them hold the same bits), and block 0 selects the experts.
constexpr int MAX_CL = 8;

__device__ __forceinline__ uint32_t cluster_rank() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
  return r;
}
__device__ __forceinline__ uint32_t cluster_blocks() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_nctarank;" : "=r"(r));
  return r;
}
// every thread of every block of the cluster; what was stored before it is visible after it
__device__ __forceinline__ void cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// store into the same shared-memory place of another block of the cluster
__device__ __forceinline__ void store_to_block(float* local, uint32_t rank, float v) {
  const uint32_t la = (uint32_t)__cvta_generic_to_shared(local);
  uint32_t ra;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ra) : "r"(la), "r"(rank));
  asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(ra), "f"(v) : "memory");
}
// the sum of one value per block; slots: MAX_CL floats of this block that nothing else uses
__device__ __forceinline__ float cluster_sum(float block_value, float* slots, uint32_t rank, uint32_t n) {
  if (threadIdx.x < n) store_to_block(slots + rank, threadIdx.x, block_value);
  __syncwarp();
  cluster_barrier();
  float t = 0.f;
  for (uint32_t i = 0; i < n; ++i) t += slots[i];
  return t;
}

// The router of one row, by its cluster: smem holds this block's columns of the row (the first of them 4 c0), then room
// for the partial logits.
template <typename TW>
__device__ __forceinline__ void route_by_cluster(const RowArgs& a, float* smem, int vec_per_block, int c0, uint32_t rank,
                                                 uint32_t CL) {
  const int H = a.H;
  // ---- router over this block's columns: a job is (group of 4 experts, strided share of the columns)
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const int E = a.E;
  constexpr int EG = 4;
  const int groups = (E + EG - 1) / EG;
  const int k = n_warps >= groups ? n_warps / groups : 1;   // warps per expert group
  const int cols = 4 * vec_per_block;
  const int r = blockIdx.x / CL, first = 4 * c0;
  const int n_valid = max(0, min(cols, H - first));          // columns of the row that this block holds
  float* part = smem + cols;                                  // [E][k]
  float* logit_slots = part + E * k;                          // [CL][E], filled in block 0 by every block
  float* s = logit_slots + MAX_CL * E;                        // [E], for more than 32 experts
  const TW* wr = (const TW*)a.wr + first;
  const bool vec = (H & 7) == 0 && (first & 7) == 0;
  for (int job = warp; job < groups * k; job += n_warps) {
    const int e0 = (job / k) * EG, sl = job % k;
    float acc[EG];
#pragma unroll
    for (int j = 0; j < EG; ++j) acc[j] = 0.f;
    if (vec) {
#pragma unroll 2
      for (int d = (sl * 32 + lane) * 8; d < n_valid; d += k * 256) {
        float wv[EG][8];
#pragma unroll
        for (int j = 0; j < EG; ++j) {
          if (e0 + j < E) {
            load_w8(wr + (size_t)(e0 + j) * H + d, wv[j]);
          } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) wv[j][i] = 0.f;
          }
        }
        const float4 x0 = ld4(smem + d), x1 = ld4(smem + d + 4);
        const float xv[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
        for (int j = 0; j < EG; ++j)
#pragma unroll
          for (int i = 0; i < 8; ++i) acc[j] = fmaf(xv[i], wv[j][i], acc[j]);
      }
    } else {
      for (int d = sl * 32 + lane; d < n_valid; d += k * 32) {
        const float xv = smem[d];
#pragma unroll
        for (int j = 0; j < EG; ++j)
          acc[j] = fmaf(xv, e0 + j < E ? to_f32(wr[(size_t)(e0 + j) * H + d]) : 0.f, acc[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < EG; ++j) {
      const float t = warp_sum(acc[j]);
      if (lane == 0 && e0 + j < E) part[(e0 + j) * k + sl] = t;
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    float t = 0.f;
    for (int i = 0; i < k; ++i) t += part[e * k + i];      // fixed order
    store_to_block(logit_slots + rank * E + e, 0, t);
  }
  __syncwarp();
  cluster_barrier();
  if (rank != 0 || warp != 0) return;
  if (a.top > 0) {                                         // softmax router limited to groups: the warp selects
    for (int e = lane; e < E; e += 32) {
      float t = 0.f;
      for (uint32_t q = 0; q < CL; ++q) t += logit_slots[q * E + e];    // fixed order
      s[e] = t;
      if (a.router_logits) a.router_logits[(size_t)r * E + e] = t;
    }
    __syncwarp();
    if (a.rule >= 2)
      select_corrected_by_warp(s, s + E, a.correction, a.rule == 3, lane, E, a.top, a.n_groups, a.keep, a.normalize, a.out_scale,
                                     a.expert_ids + (size_t)a.top * r, a.gates + (size_t)a.top * r);
    else if (a.rule == 1)
      select_sigmoid_by_warp(s, lane, E - a.extra, a.extra, a.top, a.expert_ids + (size_t)a.top * r,
                             a.gates + (size_t)a.top * r, a.aux + (size_t)(a.top + a.extra) * r);
    else
      select_topk_by_warp(s, lane, E, a.top, a.n_groups, a.keep, a.out_scale, a.expert_ids + (size_t)a.top * r,
                          a.gates + (size_t)a.top * r);
    return;
  }
  if (E <= 32) {
    float sv = -INFINITY;
    if (lane < E) {
      sv = 0.f;
      for (uint32_t q = 0; q < CL; ++q) sv += logit_slots[q * E + lane];    // fixed order
      if (a.router_logits) a.router_logits[(size_t)r * E + lane] = sv;
    }
    select_two_by_lanes(sv, lane, E, a.jitter_eps, a.expert_ids + 2 * r, a.gates + 2 * r);
    return;
  }
  if (lane != 0) return;
  for (int e = 0; e < E; ++e) {
    float t = 0.f;
    for (uint32_t q = 0; q < CL; ++q) t += logit_slots[q * E + e];
    s[e] = t;
    if (a.router_logits) a.router_logits[(size_t)r * E + e] = t;
  }
  select_two_serial(s, E, a.jitter_eps, a.expert_ids + 2 * r, a.gates + 2 * r);
}

template <int VPT, typename TW, int ST>
__global__ void __launch_bounds__(256)
row_norm_cluster_kernel(const __grid_constant__ RowArgs a, const int vec_per_block) {
  extern __shared__ float smem[];          // router only: this block's columns of the normalised row, partial logits
  __shared__ float red[32];
  __shared__ StreamWeights<ST> hw;
  __shared__ float sum_slots[MAX_CL], sq_slots[MAX_CL];
  const uint32_t rank = cluster_rank(), CL = cluster_blocks();
  const int H = a.H, n4 = H >> 2;
  const int r = blockIdx.x / CL;
  const int c0 = rank * vec_per_block;     // first vector of four columns of this block
  int col[VPT];
  bool ok[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int l = threadIdx.x + i * blockDim.x;
    col[i] = c0 + l;
    ok[i] = l < vec_per_block && col[i] < n4;
  }
  // scale and shift are weights, which no kernel writes: they are fetched while the kernel before still runs
  float4 g[VPT], b[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    g[i] = (a.gamma && ok[i]) ? ld4(a.gamma + 4 * col[i]) : make_float4(0.f, 0.f, 0.f, 0.f);
    b[i] = (a.gamma && a.beta && ok[i]) ? ld4(a.beta + 4 * col[i]) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_launch();
  if constexpr (ST > 0) load_stream_weights<ST>(hw, a);
  cluster_barrier();        // every block of the cluster runs before any of them writes into another's memory
  pdl_wait();
  const int src = a.row_index ? a.row_index[r] : r;
  float* xr = a.x + (size_t)src * (ST > 0 ? a.n_streams : 1) * H;
  float4 v[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) v[i] = ST == 0 && ok[i] ? ld4(xr + 4 * col[i]) : make_float4(0.f, 0.f, 0.f, 0.f);
  const bool pending = a.partials || a.comb_y;
  if (a.partials) {
    const float* pr = a.partials + (size_t)src * H;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      if (ok[i]) {
        for (int z0 = 0; z0 < a.n_partials; z0 += 8) {      // eight loads in flight, added in a fixed order
          float4 t[8];
#pragma unroll
          for (int u = 0; u < 8; ++u)
            t[u] = z0 + u < a.n_partials ? ld4(pr + (size_t)(z0 + u) * a.partial_stride + 4 * col[i])
                                         : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int u = 0; u < 8; ++u) add4(v[i], t[u]);
        }
        if (a.add_bias) add4(v[i], ld4(a.add_bias + 4 * col[i]));
      }
    }
  }
  if (a.comb_y) {
    float4 t[VPT];                                   // gated rows summed in the order of the choices, then added
#pragma unroll
    for (int i = 0; i < VPT; ++i) t[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < a.comb_top; ++k) {
      const float g = a.comb_gates[(size_t)a.comb_top * src + k];
      const float* y = a.comb_y + (size_t)a.comb_row_of[(size_t)a.comb_top * src + k] * H;
#pragma unroll
      for (int i = 0; i < VPT; ++i)
        if (ok[i]) fma4(t[i], g, ld4(y + 4 * col[i]));
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i)
      if (ok[i]) add4(v[i], t[i]);
  }
  if constexpr (ST > 0) {
#pragma unroll
    for (int i = 0; i < VPT; ++i)
      if (ok[i]) v[i] = stream_columns<ST>(xr + 4 * col[i], v[i], hw, a, pending);
  } else if (pending) {
#pragma unroll
    for (int i = 0; i < VPT; ++i)
      if (ok[i]) *reinterpret_cast<float4*>(xr + 4 * col[i]) = v[i];
  }
  if (!a.gamma) return;                     // only the additions were wanted (the same for every block)
  float mean = 0.f;
  if (a.mode == 0) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);   // zeros outside the block's columns
    mean = cluster_sum(block_sum(s, red), sum_slots, rank, CL) / (float)H;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    if (ok[i]) {
      const float d0 = v[i].x - mean, d1 = v[i].y - mean, d2 = v[i].z - mean, d3 = v[i].w - mean;
      ss += (d0 * d0 + d1 * d1) + (d2 * d2 + d3 * d3);
    }
  }
  const float inv = 1.0f / sqrtf(cluster_sum(block_sum(ss, red), sq_slots, rank, CL) / (float)H + a.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    if (ok[i]) {
      const int c = col[i];
      float4 y = make_float4((v[i].x - mean) * inv * g[i].x, (v[i].y - mean) * inv * g[i].y,
                             (v[i].z - mean) * inv * g[i].z, (v[i].w - mean) * inv * g[i].w);
      if (a.beta) add4(y, b[i]);
      if (a.out_f32) *reinterpret_cast<float4*>(a.out_f32 + (size_t)r * H + 4 * c) = y;
      if (a.out_bf16) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(y.x, y.y), hi = __floats2bfloat162_rn(y.z, y.w);
        uint2 pk;
        pk.x = *reinterpret_cast<const uint32_t*>(&lo);
        pk.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(a.out_bf16 + (size_t)r * H + 4 * c) = pk;
      }
      if (a.wr) *reinterpret_cast<float4*>(smem + 4 * (c - c0)) = y;
    }
  }
  if (!a.wr) return;
  route_by_cluster<TW>(a, smem, vec_per_block, c0, rank, CL);
}

// ---- norm of what is added
//   r = sum_b scale_b (sum_z partials_b[z][row] + bias_b) + sum_j g_j y[r_j];   x[row] += r / rms(r) * gamma  (no gamma: x[row] += r)
//   out = x[row], or with a convolution over time  out = x[row] + sum_d w[:, taps - 1 - d] * (the row d positions earlier)
// and on request the routing of x[row].  The convolution is for batches of single tokens: the earlier rows come from the
// request's state, taps - 1 rows, the row of position p in state row p mod (taps - 1); a thread reads the rows of its
// columns before it writes its own.
struct PostArgs : RowArgs {
  const float* part[4]; int n_part[4]; long long part_stride[4]; const float* part_bias[4]; float part_scale[4]; int n_branches;
  const float* conv_w; int taps; float* ring; long long ring_stride; const int* pos; const int* slot;
};

// four neighbouring columns of what is added to a row
__device__ __forceinline__ float4 added_columns(const PostArgs& a, int row, int c) {
  float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int b = 0; b < a.n_branches; ++b) {
    const float* p = a.part[b] + (size_t)row * a.H + 4 * c;
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int z0 = 0; z0 < a.n_part[b]; z0 += 4) {        // four loads in flight, added in a fixed order
      float4 t[4];
#pragma unroll
      for (int u = 0; u < 4; ++u)
        t[u] = z0 + u < a.n_part[b] ? ld4(p + (size_t)(z0 + u) * a.part_stride[b]) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int u = 0; u < 4; ++u) add4(y, t[u]);
    }
    if (a.part_bias[b]) add4(y, ld4(a.part_bias[b] + 4 * c));
    fma4(r, a.part_scale[b], y);
  }
  for (int k = 0; k < a.comb_top; ++k)
    fma4(r, a.comb_gates[(size_t)a.comb_top * row + k], ld4(a.comb_y + (size_t)a.comb_row_of[(size_t)a.comb_top * row + k] * a.H + 4 * c));
  return r;
}

// the new row's four columns y: stored, convolved, handed out
__device__ __forceinline__ void leave_columns(const PostArgs& a, int row, int c, float4 y) {
  *reinterpret_cast<float4*>(a.x + (size_t)row * a.H + 4 * c) = y;
  if (a.conv_w) {
    const int p = a.pos[row], R = a.taps - 1;
    float* ring = a.ring + (size_t)a.slot[row] * a.ring_stride + 4 * c;
    const float* w = a.conv_w + (size_t)4 * c * a.taps;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int d = R; d >= 0; --d) {                       // oldest first, as over prompts
      if (d > p) continue;
      const int j = R - d;
      float4 x = y;
      if (d > 0) {
        const float* q = ring + (size_t)((p - d) % R) * a.H;
        x = make_float4(q[0], q[1], q[2], q[3]);
      }
      acc.x = fmaf(w[j], x.x, acc.x); acc.y = fmaf(w[a.taps + j], x.y, acc.y);
      acc.z = fmaf(w[2 * a.taps + j], x.z, acc.z); acc.w = fmaf(w[3 * a.taps + j], x.w, acc.w);
    }
    if (R > 0) {
      float* q = ring + (size_t)(p % R) * a.H;
      q[0] = y.x; q[1] = y.y; q[2] = y.z; q[3] = y.w;
    }
    add4(y, acc);
  }
  if (a.out_f32) *reinterpret_cast<float4*>(a.out_f32 + (size_t)row * a.H + 4 * c) = y;
  if (a.out_bf16) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(y.x, y.y), hi = __floats2bfloat162_rn(y.z, y.w);
    uint2 pk;
    pk.x = *reinterpret_cast<const uint32_t*>(&lo);
    pk.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(a.out_bf16 + (size_t)row * a.H + 4 * c) = pk;
  }
}

template <int VPT, typename TW>
__global__ void __launch_bounds__(1024)
row_post_kernel(const __grid_constant__ PostArgs a) {
  extern __shared__ float smem[];
  __shared__ float red[32];
  pdl_launch();
  pdl_wait();
  const int n4 = a.H >> 2, row = blockIdx.x;
  const float* xr = a.x + (size_t)row * a.H;
  float4 x[VPT], v[VPT];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    x[i] = v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < n4) {
      x[i] = ld4(xr + 4 * c);
      v[i] = added_columns(a, row, c);
    }
    ss += (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
  }
  float inv = 1.f;
  if (a.gamma) inv = 1.0f / sqrtf(block_sum(ss, red) / (float)a.H + a.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c < n4) {
      const float4 g = a.gamma ? ld4(a.gamma + 4 * c) : make_float4(1.f, 1.f, 1.f, 1.f);
      const float4 y = make_float4(x[i].x + v[i].x * inv * g.x, x[i].y + v[i].y * inv * g.y, x[i].z + v[i].z * inv * g.z,
                                   x[i].w + v[i].w * inv * g.w);
      if (a.wr) *reinterpret_cast<float4*>(smem + 4 * c) = y;
      leave_columns(a, row, c, y);
    }
  }
  if (a.wr) route_by_block<TW>(a, smem);
}

template <int VPT, typename TW>
__global__ void __launch_bounds__(256)
row_post_cluster_kernel(const __grid_constant__ PostArgs a, const int vec_per_block) {
  extern __shared__ float smem[];
  __shared__ float red[32];
  __shared__ float sq_slots[MAX_CL];
  const uint32_t rank = cluster_rank(), CL = cluster_blocks();
  const int n4 = a.H >> 2, row = blockIdx.x / CL, c0 = rank * vec_per_block;
  float4 g[VPT], x[VPT], v[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {           // a weight, which no kernel writes: fetched while the kernel before still runs
    const int l = threadIdx.x + i * blockDim.x, c = c0 + l;
    g[i] = a.gamma && l < vec_per_block && c < n4 ? ld4(a.gamma + 4 * c) : make_float4(1.f, 1.f, 1.f, 1.f);
  }
  pdl_launch();
  cluster_barrier();        // every block of the cluster runs before any of them writes into another's memory
  pdl_wait();
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int l = threadIdx.x + i * blockDim.x, c = c0 + l;
    x[i] = v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (l < vec_per_block && c < n4) {
      x[i] = ld4(a.x + (size_t)row * a.H + 4 * c);
      v[i] = added_columns(a, row, c);
    }
    ss += (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
  }
  float inv = 1.f;
  if (a.gamma) inv = 1.0f / sqrtf(cluster_sum(block_sum(ss, red), sq_slots, rank, CL) / (float)a.H + a.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int l = threadIdx.x + i * blockDim.x, c = c0 + l;
    if (l < vec_per_block && c < n4) {
      const float4 y = make_float4(x[i].x + v[i].x * inv * g[i].x, x[i].y + v[i].y * inv * g[i].y,
                                   x[i].z + v[i].z * inv * g[i].z, x[i].w + v[i].w * inv * g[i].w);
      if (a.wr) *reinterpret_cast<float4*>(smem + 4 * l) = y;
      leave_columns(a, row, c, y);
    }
  }
  if (a.wr) route_by_cluster<TW>(a, smem, vec_per_block, c0, rank, CL);
}

template <typename Args>
int launch_row(void (*kernel)(Args), bool& configured, const Args& a, int rows, int threads, size_t smem, cudaStream_t stream) {
  if (smem > 48 * 1024 && !configured) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return fail("row_norm: cannot raise shared memory: %s", cudaGetErrorString(e));
    configured = true;
  }
  launch_pdl(kernel, dim3(rows), dim3(threads), smem, stream, a);
  return check_launch("row_norm");
}

template <typename Args>
int launch_row_cluster(void (*kernel)(Args, int), const Args& a, int rows, int cl, int vec_per_block, int threads, size_t smem,
                       cudaStream_t stream) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(rows * cl);
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = cl;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  cudaLaunchKernelEx(&cfg, kernel, a, vec_per_block);
  return check_launch("row_norm (cluster)");
}

// Streams of any width: x brought up to date with what is pending (if it names mixing weights), u [rows, H] (or null) the
// sum of the streams weighted by gather.  One block per row.
__global__ void stream_update_kernel(const __grid_constant__ RowArgs a, float* __restrict__ u) {
  __shared__ StreamWeights<MAX_STREAMS> w;
  pdl_launch();
  load_stream_weights<MAX_STREAMS>(w, a);
  __syncthreads();
  pdl_wait();
  const int src = a.row_index ? a.row_index[blockIdx.x] : blockIdx.x;
  const int H = a.H, n = a.n_streams;
  const bool pending = a.partials || a.comb_y;
  float* xr = a.x + (size_t)src * n * H;
  for (int c = threadIdx.x; c < H; c += blockDim.x) {
    float r = 0.f;
    for (int z = 0; z < a.n_partials; ++z) r += a.partials[(size_t)z * a.partial_stride + (size_t)src * H + c];
    if (a.add_bias) r += a.add_bias[c];
    float e = 0.f;
    for (int k = 0; k < a.comb_top; ++k)
      e = fmaf(a.comb_gates[(size_t)a.comb_top * src + k], a.comb_y[(size_t)a.comb_row_of[(size_t)a.comb_top * src + k] * H + c], e);
    r += e;
    float x[MAX_STREAMS], g = 0.f;
    for (int s = 0; s < n; ++s) x[s] = xr[(size_t)s * H + c];
    for (int t = 0; t < n; ++t) {
      float v = x[t];
      if (pending) {
        v = 0.f;
        for (int s = 0; s < n; ++s) v = fmaf(w.mix[s * n + t], x[s], v);
        v = fmaf(w.spread[t], r, v);
        if (a.store) xr[(size_t)t * H + c] = v;
      }
      g = fmaf(w.gather[t], v, g);
    }
    if (u) u[(size_t)blockIdx.x * H + c] = g;
  }
}

int g_cluster_rows = 16;      // up to this many rows a cluster of blocks shares each row; 0: never

// How rows of H numbers are worked: `cl` blocks a row (1: one block), threads a block, vectors of four a thread, shared memory.
// E > 0: with a router.  threads 0: the row and the router do not fit.
struct RowPlan { int cl, vec_per_block, threads, vpt; size_t smem; };

RowPlan plan_rows(int rows, int H, int E, bool streams) {
  const int n4 = H / 4, groups = (E + 3) / 4;
  RowPlan p = {};
  // a handful of rows: a cluster of blocks per row
  // (measured on a decode step of rows of 4,096: 1, 8 and 16 rows gain 3.7, 1.8 and 1.0 % of the step; 32 rows
  // lose 1.2 %, also with clusters of four: with that many blocks the barriers cost more than the blocks gain)
  p.cl = n4 >= 512 ? 8 : (n4 >= 256 ? 4 : (n4 >= 128 ? 2 : 1));
  if (p.cl > 1 && rows <= g_cluster_rows) {
    p.vec_per_block = (((n4 + p.cl - 1) / p.cl) + 1) & ~1;       // even: a block's columns start on 32 bytes
    p.threads = ((p.vec_per_block + 31) / 32) * 32;
    if (p.threads > 256) p.threads = 256;
    p.vpt = (p.vec_per_block + p.threads - 1) / p.threads;
    const int n_warps = p.threads / 32;
    const int k = E ? (n_warps >= groups ? n_warps / groups : 1) : 0;
    p.smem = E ? (size_t)(4 * p.vec_per_block + E * k + MAX_CL * E + 2 * E) * sizeof(float) : 0;
    if (p.smem <= 48 * 1024 && p.vpt <= MAX_VPT) return p;
  }
  // few rows: a wide block per row (more warps share the router's rows); many rows: narrow blocks
  // with four vectors per thread, so that several blocks fit an SM and hide each other's latency
  p.cl = 1;
  p.threads = rows < 148 ? ((n4 + 31) / 32) * 32 : ((n4 / 4 + 31) / 32) * 32;
  if (streams && rows >= 148) p.threads = ((n4 + 31) / 32) * 32;      // the streams' columns already are several loads a thread
  if (p.threads > 1024) p.threads = 1024;
  if (p.threads < 32) p.threads = 32;
  if (E && p.threads < 128) p.threads = 128;             // a few warps for the router's dot products
  p.vpt = (n4 + p.threads - 1) / p.threads;
  const int n_warps = p.threads / 32;
  const int k = E ? (n_warps >= groups ? n_warps / groups : 1) : 0;
  p.smem = E ? (size_t)(H + E * k) * sizeof(float) : 0;
  if (p.smem > 200 * 1024) p.threads = 0;
  return p;
}

template <int VPT, typename TW, int ST>
int row_norm_form(const RowArgs& a, int rows, const RowPlan& p, cudaStream_t stream) {
  static bool configured = false;   // per instantiation
  return p.cl > 1 ? launch_row_cluster(row_norm_cluster_kernel<VPT, TW, ST>, a, rows, p.cl, p.vec_per_block, p.threads, p.smem, stream)
                  : launch_row(row_norm_kernel<VPT, TW, ST>, configured, a, rows, p.threads, p.smem, stream);
}

template <int VPT, typename TW>
int row_post_form(const PostArgs& a, int rows, const RowPlan& p, cudaStream_t stream) {
  static bool configured = false;
  return p.cl > 1 ? launch_row_cluster(row_post_cluster_kernel<VPT, TW>, a, rows, p.cl, p.vec_per_block, p.threads, p.smem, stream)
                  : launch_row(row_post_kernel<VPT, TW>, configured, a, rows, p.threads, p.smem, stream);
}

// 0 if the row kernels can route by these numbers
int check_router(const void* wr, int H, int E, int top, int n_groups, int keep, int rule, int extra, const float* aux) {
  if (E < (top > 0 ? 1 : 2) || E > MAX_E) return fail("row_norm: %d experts (up to %d)", E, MAX_E);
  if (rule == 1) {
    if (top < 1 || top > ROUTER_MAX_TOP || extra < 0 || top > E - extra || !aux)
      return fail("row_norm: a sigmoid router choosing %d of %d experts (%d gate rows) is not supported", top, E - extra, extra);
  } else if (rule != 0 && rule != 2 && rule != 3) {
    return fail("row_norm: unknown router rule %d", rule);
  } else if (rule >= 2 && (top < 1 || 2 * E > H)) {
    return fail("row_norm: a router with corrected choice scores needs top >= 1 and rows of at least twice the %d experts", E);
  } else if (top > 0 && (top > ROUTER_MAX_TOP || top > E || n_groups < 1 || n_groups > 64 || E % n_groups || keep < 1 ||
                        keep > n_groups || keep * (E / n_groups) < top))
    return fail("row_norm: %d of %d experts from %d of %d groups is not supported", top, E, keep, n_groups);
  if ((uintptr_t)wr & 15) return fail("row_norm: router weights must be 16-byte aligned");
  return 0;
}
}  // namespace

// For measurements and tests: the largest number of rows that run with a cluster of blocks per row (0: none).
extern "C" int flint_row_norm_set_cluster_rows(int rows) {
  g_cluster_rows = rows < 0 ? 0 : rows;
  return 0;
}

// x [T, H] float32 residual stream, updated in place if anything is pending.
// rows: number of output rows (T, or the length of row_index if given; then x rows are gathered).
// pending: partials [n_partials][T][H] (stride partial_stride floats) + add_bias [H]; and/or
//          comb_y [comb_top T, H] with comb_row_of [T, comb_top] and comb_gates [T, comb_top].
// gamma NULL: only apply the pending additions.  wr != NULL (router weights [E, H], bf16 or f32):
// also fill expert_ids [rows, 2] and gates [rows, 2] (and router_logits [rows, E] if given); then row_index
// must be NULL.  top > 0: the router is a softmax limited to groups (`keep` of `n_groups`, `top` experts, gates times
// out_scale) and expert_ids and gates are [rows, top]; top == 0: sparsemixer top-2.  rule 1: a sigmoid router over the
// first E - extra rows of wr (the `top` largest scores, given as they are in gates); the last `extra` rows are gates of
// always-on parts, and aux [rows, top + extra] gets 1 for the chosen experts and those rows' sigmoids.  rule 2: a sigmoid
// router limited to groups: choice scores sigmoid + correction [E] (or NULL), a group scores as the sum of its two
// largest, `top` experts of the `keep` best of `n_groups` groups; gates the chosen sigmoids, over their sum if
// `normalize`, times out_scale.  rule 3: the same with softmax scores.
// n_streams > 0: x is [T, n_streams, H]; what is pending goes into the streams by mix [n_streams, n_streams] ([from, to])
// and spread [n_streams], and the norm reads their sum weighted by gather [n_streams].  With row_index the streams are
// brought up to date for the norm only, not in memory.
extern "C" int flint_row_norm(float* x, const int* row_index, int rows, int H, const float* partials,
                              int n_partials, long long partial_stride, const float* add_bias,
                              const float* comb_y, const int* comb_row_of, const float* comb_gates, int comb_top,
                              const float* gamma, const float* beta, float eps, int mode, float* out_f32,
                              void* out_bf16, const void* wr, int w_dtype, int E, float jitter_eps,
                              int* expert_ids, float* gates, float* router_logits, int top, int n_groups, int keep,
                              float out_scale, int rule, int extra, float* aux, const float* correction, int normalize,
                              int n_streams, const float* mix, const float* spread, const float* gather,
                              cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || (H & 3) || H > 4 * 1024 * MAX_VPT) return fail("row_norm: width %d (multiples of 4 up to %d)", H, 4096 * MAX_VPT);
  if (gamma && !out_f32 && !out_bf16 && !wr) return fail("row_norm: no output given");
  if (mode != 0 && mode != 1) return fail("row_norm: unknown mode %d", mode);
  if (comb_y && comb_top < 1) return fail("row_norm: %d expert rows a token", comb_top);
  if (wr) {
    const int bad = check_router(wr, H, E, top, n_groups, keep, rule, extra, aux);
    if (bad) return bad;
  }
  if (wr && (row_index || !gamma || !expert_ids || !gates)) return fail("row_norm: the router needs a norm and all rows");
  if (n_streams < 0 || n_streams > FUSED_STREAMS) return fail("row_norm: %d streams (up to %d)", n_streams, FUSED_STREAMS);
  if (n_streams && (partials || comb_y) && (!mix || !spread)) return fail("row_norm: what is pending needs the streams' mixing weights");
  if (n_streams && gamma && !gather) return fail("row_norm: the norm of several streams needs their weights");
  RowArgs a;
  a.n_streams = n_streams; a.mix = mix; a.spread = spread; a.gather = gather; a.store = row_index == nullptr;
  a.x = x; a.row_index = row_index;
  a.partials = partials; a.n_partials = n_partials; a.partial_stride = partial_stride; a.add_bias = add_bias;
  a.comb_y = comb_y; a.comb_row_of = comb_row_of; a.comb_gates = comb_gates; a.comb_top = comb_top;
  a.gamma = gamma; a.beta = beta; a.eps = eps; a.mode = mode;
  a.out_f32 = out_f32; a.out_bf16 = (__nv_bfloat16*)out_bf16;
  a.wr = wr; a.E = E; a.jitter_eps = jitter_eps; a.expert_ids = expert_ids; a.gates = gates;
  a.top = wr ? top : 0; a.n_groups = n_groups; a.keep = keep; a.out_scale = out_scale;
  a.router_logits = wr ? router_logits : nullptr;
  a.rule = wr ? rule : 0; a.extra = extra; a.aux = aux;
  a.correction = correction; a.normalize = normalize;
  a.H = H;
  const RowPlan plan = plan_rows(rows, H, wr ? E : 0, n_streams > 0);
  if (!plan.threads) return fail("row_norm: width %d is too large for the fused router", H);
#define GOS(V, S) (wr && w_dtype == FLINT_BF16 ? row_norm_form<V, __nv_bfloat16, S>(a, rows, plan, stream) : row_norm_form<V, float, S>(a, rows, plan, stream))
#define GO(V) (n_streams ? GOS(V, FUSED_STREAMS) : GOS(V, 0))
  switch (plan.vpt) {
    case 1: return GO(1);
    case 2: return GO(2);
    case 3: case 4: return GO(4);
    default: return fail("row_norm: width %d is too large", H);
  }
#undef GO
#undef GOS
}

// x [T, H] float32 += what is pending, divided by its root mean square and scaled by gamma [H] (NULL: as it is), in place.
// Pending: n_branches (up to 4) products left as partial sums, [n_part][T][H] with a stride, a bias [H] (or NULL) and a scale
// each; and/or expert rows as in flint_row_norm.  out_f32 / out_bf16 [T, H] (or NULL) receive the new rows, or, with conv_w
// [H, taps], the new rows plus their convolution over time: then every row is one request's only token, ring [slots, >= (taps
// - 1) H] (a row stride) holds its last taps - 1 rows and receives the new one.  wr != NULL: the routing of the new rows, as in
// flint_row_norm.
extern "C" int flint_row_post(float* x, int rows, int H, int n_branches, const float* const* partials, const int* n_partials,
                              const long long* strides, const float* const* bias, const float* scales, const float* comb_y,
                              const int* comb_row_of, const float* comb_gates, int comb_top, const float* gamma, float eps,
                              float* out_f32, void* out_bf16, const float* conv_w, int taps, float* ring, long long ring_stride,
                              const int* pos, const int* slot, const void* wr, int w_dtype, int E, int* expert_ids, float* gates,
                              float* router_logits, int top, int n_groups, int keep, float out_scale, int rule, int extra,
                              float* aux, const float* correction, int normalize, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || (H & 3) || H > 4 * 1024 * MAX_VPT) return fail("row_post: width %d (multiples of 4 up to %d)", H, 4096 * MAX_VPT);
  if (n_branches < 0 || n_branches > 4) return fail("row_post: %d branches are not supported (up to 4)", n_branches);
  if (comb_y && comb_top < 1) return fail("row_post: %d expert rows a token", comb_top);
  if (conv_w && (taps < 1 || taps > 64)) return fail("row_post: %d taps are not supported (1 to 64)", taps);
  if (conv_w && taps > 1 && (!ring || !pos || !slot)) return fail("row_post: a convolution over time needs the requests' state");
  if (wr && conv_w) return fail("row_post: rows are routed or convolved, not both");
  if (wr) {
    const int bad = check_router(wr, H, E, top, n_groups, keep, rule, extra, aux);
    if (bad) return bad;
    if (top < 1 || !expert_ids || !gates) return fail("row_post: the router needs its outputs");
  }
  PostArgs a = {};
  a.x = x; a.H = H;
  a.n_branches = n_branches;
  for (int b = 0; b < n_branches; ++b) {
    a.part[b] = partials[b]; a.n_part[b] = n_partials[b]; a.part_stride[b] = strides[b]; a.part_bias[b] = bias[b];
    a.part_scale[b] = scales[b];
  }
  a.comb_y = comb_y; a.comb_row_of = comb_row_of; a.comb_gates = comb_gates; a.comb_top = comb_y ? comb_top : 0;
  a.gamma = gamma; a.eps = eps; a.mode = 1;
  a.out_f32 = out_f32; a.out_bf16 = (__nv_bfloat16*)out_bf16;
  a.conv_w = conv_w; a.taps = taps; a.ring = ring; a.ring_stride = ring_stride; a.pos = pos; a.slot = slot;
  a.wr = wr; a.E = E; a.expert_ids = expert_ids; a.gates = gates; a.router_logits = wr ? router_logits : nullptr;
  a.top = wr ? top : 0; a.n_groups = n_groups; a.keep = keep; a.out_scale = out_scale;
  a.rule = wr ? rule : 0; a.extra = extra; a.aux = aux; a.correction = correction; a.normalize = normalize;
  const RowPlan plan = plan_rows(rows, H, wr ? E : 0, false);
  if (!plan.threads) return fail("row_post: width %d is too large for the fused router", H);
#define GO(V) (wr && w_dtype == FLINT_BF16 ? row_post_form<V, __nv_bfloat16>(a, rows, plan, stream) : row_post_form<V, float>(a, rows, plan, stream))
  switch (plan.vpt) {
    case 1: return GO(1);
    case 2: return GO(2);
    case 3: case 4: return GO(4);
    default: return fail("row_post: width %d is too large", H);
  }
#undef GO
}

// The streams' part of flint_row_norm as a kernel of its own, for widths and numbers of streams that one does not take: x [T, n_streams, H]
// updated in place (not with row_index), u [rows, H] the norm's input (or null).
extern "C" int flint_stream_update(float* x, const int* row_index, int rows, int H, const float* partials, int n_partials,
                                   long long partial_stride, const float* add_bias, const float* comb_y,
                                   const int* comb_row_of, const float* comb_gates, int comb_top, int n_streams,
                                   const float* mix, const float* spread, const float* gather, float* u,
                                   cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (n_streams < 1 || n_streams > MAX_STREAMS) return fail("stream_update: %d streams (up to %d)", n_streams, MAX_STREAMS);
  if ((partials || comb_y) && (!mix || !spread)) return fail("stream_update: what is pending needs the streams' mixing weights");
  if (u && !gather) return fail("stream_update: the sum of the streams needs their weights");
  if (comb_y && comb_top < 1) return fail("stream_update: %d expert rows a token", comb_top);
  RowArgs a = {};
  a.x = x; a.row_index = row_index; a.H = H;
  a.partials = partials; a.n_partials = partials ? n_partials : 0; a.partial_stride = partial_stride; a.add_bias = partials ? add_bias : nullptr;
  a.comb_y = comb_y; a.comb_row_of = comb_row_of; a.comb_gates = comb_gates; a.comb_top = comb_y ? comb_top : 0;
  a.n_streams = n_streams; a.mix = mix; a.spread = spread; a.gather = gather; a.store = row_index == nullptr;
  launch_pdl(stream_update_kernel, dim3(rows), dim3(H >= 512 ? 256 : 128), 0, stream, a, u);
  return check_launch("stream_update");
}

extern "C" const char* flint_row_fused_last_error() { return g_error; }
