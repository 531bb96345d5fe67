// The token table beside the layers, for steps of few rows, in one launch with the row steps around it:
//
//   x += post(y)                                     what the sublayer before left (see row_rms_kernel)
//   g  = gelu(gate x) * e                            e: the layer's part of the row of the token's table
//   x += post_side(proj g),   h = next norm of x
//
// A cluster of CTAs owns one row.  Every CTA forms the whole row x for itself, multiplies its share of the gate's rows,
// stores the results into every CTA's shared memory, then finishes its share of the channels; the two root mean squares are sums
// over the cluster.  Weights and constants are requested ahead of the dependency wait.  Remote memory is only written, and never
// behind the last cluster barrier, so that a CTA may leave as soon as it is done.
// Steps of many rows, and matrices that sixteen SMs would take long to read, take separate projections with row_rms_kernel in
// between.
#include <cooperative_groups.h>

#include <algorithm>

#include "pi_layered.cuh"

namespace cg = cooperative_groups;

namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32;
constexpr int kMaxCluster = 16;
constexpr int kAhead = 8;             // 16-byte loads a thread has in flight
constexpr size_t kMaxBytes = 1536 * 1024;   // of both matrices (at 1 MB the one launch saves 3 us, at 4 MB it loses 6)

enum SideSource { kResult, kExperts };

struct SideParams {
  float* x;
  int width, dim, per_gate, per_channel;   // gate rows and channels of a CTA
  const float* y;
  size_t y_stride;
  pi_expert_sum e;
  const float* post_w;
  float post_eps;
  const __nv_bfloat16 *gate, *proj;
  int ld_gate, ld_proj;
  pi_token_table table;
  const float *side_w, *next_w;
  float side_eps, next_eps;
  void* h;
  size_t ld_h;
  int h_bf16;
};

__device__ __forceinline__ float4 expert_value4(const pi_expert_sum& e, size_t i) {
  if (!e.y_bf16) return *reinterpret_cast<const float4*>(static_cast<const float*>(e.y) + i);
  const uint2 u = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(e.y) + i);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ float4 fma4(float a, float4 b, float4 c) {
  return make_float4(fmaf(a, b.x, c.x), fmaf(a, b.y, c.y), fmaf(a, b.z, c.z), fmaf(a, b.w, c.w));
}
__device__ __forceinline__ float dot4(float4 v) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))); }
__device__ __forceinline__ void fma8(uint4 w, const float* x, float& a) {   // eight bf16 weights
  const float4 lo = *reinterpret_cast<const float4*>(x), hi = *reinterpret_cast<const float4*>(x + 4);
  a = fmaf(__uint_as_float(w.x << 16), lo.x, a);
  a = fmaf(__uint_as_float(w.x & 0xffff0000u), lo.y, a);
  a = fmaf(__uint_as_float(w.y << 16), lo.z, a);
  a = fmaf(__uint_as_float(w.y & 0xffff0000u), lo.w, a);
  a = fmaf(__uint_as_float(w.z << 16), hi.x, a);
  a = fmaf(__uint_as_float(w.z & 0xffff0000u), hi.y, a);
  a = fmaf(__uint_as_float(w.w << 16), hi.z, a);
  a = fmaf(__uint_as_float(w.w & 0xffff0000u), hi.w, a);
}
// Sum over the CTA, the same bits in every thread.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = pi_warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) t += red[w];
  return t;
}

template <SideSource SRC>
__global__ void __launch_bounds__(kThreads) token_side_kernel(const SideParams p) {
  extern __shared__ __align__(16) float sm[];
  cg::cluster_group cluster = cg::this_cluster();
  const int cs = (int)cluster.num_blocks(), rank = (int)cluster.block_rank(), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int row = (int)(blockIdx.x / cs), W = p.width;
  const int d0 = min(p.dim, rank * p.per_gate), d1 = min(p.dim, d0 + p.per_gate), c0 = min(W, rank * p.per_channel), c1 = min(W, c0 + p.per_channel);
  float* xs = sm;                                     // [ld_gate] the row, zeros behind it
  float* g = xs + p.ld_gate;                          // [ld_proj] gate results, zeros behind them
  float* yrow = g + p.ld_proj;                        // [W] the result of the sublayer before
  float* wrow = yrow + W;                             // [W] post_w
  float* ys = wrow + W;                               // [per_channel]
  float* ws = ys + p.per_channel;                     // [2][per_channel] side_w, next_w of the CTA's channels
  __shared__ float red[kWarps], ss_all[2][kMaxCluster];

  // ---- constants, ahead of the wait ----------------------------------------------------------------------------------
  uint4 gw[kAhead];                                   // the first of this warp's gate rows
  const __nv_bfloat16* grow = p.gate + (size_t)min(d0 + warp, p.dim - 1) * p.ld_gate;
#pragma unroll
  for (int j = 0; j < kAhead; ++j) gw[j] = __ldg(reinterpret_cast<const uint4*>(grow + min(lane * 8 + 256 * j, p.ld_gate - 8)));
  int lpr = 32;                                       // lanes per row of proj
  while (lpr > 1 && (lpr >> 1) * 8 >= p.ld_proj) lpr >>= 1;
  const int grp = tid / lpr, gl = tid - grp * lpr, groups = kThreads / lpr;
  auto proj_at = [&](int i, int k) { return reinterpret_cast<const uint4*>(p.proj + (size_t)min(c0 + i, W - 1) * p.ld_proj + min(k, p.ld_proj - 8)); };
  uint4 pw[kAhead];                                   // the first columns of this group's first rows of proj
#pragma unroll
  for (int j = 0; j < kAhead; ++j) pw[j] = __ldg(proj_at(grp + j * groups, gl * 8));
  for (int i = tid; i < c1 - c0; i += kThreads) {
    ws[i] = __ldg(p.side_w + c0 + i);
    ws[p.per_channel + i] = p.h ? __ldg(p.next_w + c0 + i) : 0.f;
  }
  for (int i = tid * 4; i < W; i += kThreads * 4) *reinterpret_cast<float4*>(wrow + i) = __ldg(reinterpret_cast<const float4*>(p.post_w + i));
  for (int i = tid; i < p.ld_proj; i += kThreads) g[i] = 0.f;
  for (int i = W + tid; i < p.ld_gate; i += kThreads) xs[i] = 0.f;
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");   // every CTA runs, its g is empty; awaited before the first remote store
  pi_grid_dependency_wait();

  // ---- the row ----------------------------------------------------------------------------------------------------------
  const float* x = p.x + (size_t)row * W;
  const float e_mine = pi_table_value(p.table, row, min(d0 + warp + kWarps * lane, p.dim - 1));   // lane j: this warp's gate row number j
  float ss = 0.f;
  if (SRC == kResult) {
    for (int i = tid * 4; i < W; i += kThreads * 4) {
      const float4 a = *reinterpret_cast<const float4*>(x + i), v = *reinterpret_cast<const float4*>(p.y + (size_t)row * p.y_stride + i);
      *reinterpret_cast<float4*>(xs + i) = a;
      *reinterpret_cast<float4*>(yrow + i) = v;
      ss += dot4(v);
    }
  } else {
    const pi_expert_sum& e = p.e;
    const float gate = e.shared_gate ? pi_sigmoid(e.shared_gate[(size_t)row * e.shared_gate_stride]) : 1.f;
    for (int i = tid * 4; i < W; i += kThreads * 4) {
      const float4 a = *reinterpret_cast<const float4*>(x + i);
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (e.shared) v = fma4(gate, *reinterpret_cast<const float4*>(e.shared + (size_t)row * e.shared_stride + i), v);
      for (int k0 = 0; k0 < e.top; k0 += kAhead) {
        float4 z[kAhead];
        float w[kAhead];
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
          const int pair = row * e.top + min(k0 + k, e.top - 1);
          w[k] = e.weights[pair];
          z[k] = expert_value4(e, (size_t)(e.place ? e.place[pair] : pair) * e.y_stride + i);
        }
#pragma unroll
        for (int k = 0; k < kAhead; ++k)
          if (k0 + k < e.top) v = fma4(w[k], z[k], v);
      }
      *reinterpret_cast<float4*>(xs + i) = a;
      *reinterpret_cast<float4*>(yrow + i) = v;
      ss += dot4(v);
    }
  }
  const float inv1 = 1.0f / sqrtf(block_sum(ss, red) / (float)W + p.post_eps);
  for (int i = tid; i < W; i += kThreads) xs[i] = fmaf(yrow[i] * inv1, wrow[i], xs[i]);
  __syncthreads();

  // ---- gate: a warp per row ------------------------------------------------------------------------------------------------
  bool waited = false;
  for (int d = d0 + warp, j0 = 0; d < d1; d += kWarps, ++j0) {
    float acc = 0.f;
    const __nv_bfloat16* w = p.gate + (size_t)d * p.ld_gate;
    for (int k0 = 0; k0 < p.ld_gate; k0 += 256 * kAhead) {
      if (k0 > 0 || j0 > 0) {
#pragma unroll
        for (int j = 0; j < kAhead; ++j) gw[j] = __ldg(reinterpret_cast<const uint4*>(w + min(k0 + lane * 8 + 256 * j, p.ld_gate - 8)));
      }
#pragma unroll
      for (int j = 0; j < kAhead; ++j) {
        const int k = k0 + lane * 8 + 256 * j;
        if (k < p.ld_gate) fma8(gw[j], xs + k, acc);
      }
    }
    const float e = j0 < 32 ? __shfl_sync(0xffffffffu, e_mine, j0) : pi_table_value(p.table, row, d);
    const float v = pi_gelu_tanh(pi_warp_sum(acc)) * e;
    if (!waited) {
      asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
      waited = true;
    }
    if (lane < cs) cluster.map_shared_rank(g, lane)[d] = v;
  }
  if (!waited) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
  cluster.sync();

  // ---- proj: lpr lanes per row -----------------------------------------------------------------------------------------------
  const int mine = c1 - c0;
  for (int i0 = grp; i0 - grp < mine; i0 += kAhead * groups) {      // the same number of rounds for every thread
    float acc[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) acc[j] = 0.f;
    for (int k = gl * 8; k - gl * 8 < p.ld_proj; k += lpr * 8) {
      if (i0 != grp || k != gl * 8) {
#pragma unroll
        for (int j = 0; j < kAhead; ++j) pw[j] = __ldg(proj_at(i0 + j * groups, k));
      }
      if (k < p.ld_proj) {
#pragma unroll
        for (int j = 0; j < kAhead; ++j) fma8(pw[j], g + k, acc[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      for (int o = lpr >> 1; o > 0; o >>= 1) acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], o);
    if (gl == 0) {
#pragma unroll
      for (int j = 0; j < kAhead; ++j)
        if (i0 + j * groups < mine) ys[i0 + j * groups] = acc[j];
    }
  }
  __syncthreads();

  // ---- both norms: sums over the cluster ---------------------------------------------------------------------------------------
  auto cluster_sum = [&](float v, int which) {
    v = block_sum(v, red);
    if (tid < cs) cluster.map_shared_rank(&ss_all[0][0], tid)[which * kMaxCluster + rank] = v;
    cluster.sync();
    v = 0.f;
    for (int c = 0; c < cs; ++c) v += ss_all[which][c];
    return v;
  };
  ss = 0.f;
  for (int i = tid; i < mine; i += kThreads) ss = fmaf(ys[i], ys[i], ss);
  const float inv2 = 1.0f / sqrtf(cluster_sum(ss, 0) / (float)W + p.side_eps);
  ss = 0.f;
  for (int i = tid; i < mine; i += kThreads) {
    const float v = fmaf(ys[i] * inv2, ws[i], xs[c0 + i]);
    ys[i] = v;
    p.x[(size_t)row * W + c0 + i] = v;
    ss = fmaf(v, v, ss);
  }
  if (!p.h) return;                                   // for every CTA alike
  const float inv3 = 1.0f / sqrtf(cluster_sum(ss, 1) / (float)W + p.next_eps);
  const size_t at = (size_t)row * p.ld_h + c0;
  for (int i = tid; i < mine; i += kThreads) {
    const float v = ys[i] * inv3 * ws[p.per_channel + i];
    if (p.h_bf16) static_cast<__nv_bfloat16*>(p.h)[at + i] = __float2bfloat16_rn(v);
    else static_cast<float*>(p.h)[at + i] = v;
  }
}

typedef void (*SideKernel)(const SideParams);

cudaError_t prepare(pi_ctx* ctx, SideKernel k, size_t smem, pi_smem_grant& g) {
  if (g.of(ctx) == 0) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    if (e != cudaSuccess) return e;
    g.of(ctx) = kSmemFree;
  }
  if (smem <= g.of(ctx)) return cudaSuccess;
  g.of(ctx) = smem;
  return cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

int max_clusters(pi_ctx* ctx, SideKernel k, size_t smem, int size) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(size);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = smem;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = size;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  int n = 0;
  if (cudaOccupancyMaxActiveClusters(&n, k, &cfg) != cudaSuccess) {
    cudaGetLastError();
    n = 0;
  }
  return n;
}

SideParams sizes(const pi_token_side& s, int width, int cs) {
  SideParams p = {};
  p.width = width;
  p.dim = (int)s.gate->rows;
  p.ld_gate = (int)s.gate->ld;
  p.ld_proj = (int)s.proj->ld;
  p.per_gate = (p.dim + cs - 1) / cs;
  p.per_channel = ((width + cs - 1) / cs + 3) / 4 * 4;
  return p;
}
size_t smem_of(const SideParams& p) { return sizeof(float) * ((size_t)p.ld_gate + p.ld_proj + 2 * (size_t)p.width + 3 * (size_t)p.per_channel); }

}  // namespace

bool pi_token_side_usable(const pi_ctx* ctx, const pi_token_side& s, int rows, int width) {
  return rows <= kSideRows && width % 4 == 0 && 2 * (s.gate->rows * s.gate->ld + s.proj->rows * s.proj->ld) <= kMaxBytes && s.gate->kind == PI_BF16 && s.proj->kind == PI_BF16 && smem_of(sizes(s, width, 8)) + 4096 <= ctx->smem_optin;
}

pi_status pi_launch_token_side(pi_ctx* ctx, const pi_token_side& s, const pi_row_norm& n) {
  static pi_smem_grant granted[2];
  static struct {
    size_t smem = 0;
    int clusters = 0;
  } wide[2][64];                       // clusters of 16 the device holds
  PI_REQUIRE(ctx, pi_token_side_usable(ctx, s, n.rows, n.width) && n.rms && !n.pick && !n.table, "this step does not fit the fused kernel");
  PI_REQUIRE(ctx, !n.experts || (n.experts->y_stride % 4 == 0 && n.experts->shared_stride % 4 == 0 && !n.experts->scale), "the experts' rows do not fit the fused kernel");
  PI_REQUIRE(ctx, (n.experts || (n.y && n.y_stride % 4 == 0)) && n.post.w && (!n.h || n.norm.w), "operands are missing");
  const int pick = n.experts != nullptr;
  const SideKernel k = pick ? token_side_kernel<kExperts> : token_side_kernel<kResult>;
  const size_t smem8 = smem_of(sizes(s, n.width, 8));
  PI_CUDA(ctx, prepare(ctx, k, smem8, granted[pick]));
  auto& w = wide[pick][(unsigned)ctx->device & 63u];
  if (w.smem != smem8) w = {smem8, max_clusters(ctx, k, smem8, kMaxCluster)};
  const int cs = n.rows <= w.clusters ? kMaxCluster : 8;
  SideParams p = sizes(s, n.width, cs);
  p.x = n.x;
  p.y = n.y;
  p.y_stride = n.y_stride;
  if (n.experts) p.e = *n.experts;
  p.post_w = n.post.w;
  p.post_eps = n.post.eps;
  p.gate = static_cast<const __nv_bfloat16*>(s.gate->w);
  p.proj = static_cast<const __nv_bfloat16*>(s.proj->w);
  p.table = s.table;
  p.side_w = s.post.w;
  p.side_eps = s.post.eps;
  p.next_w = n.norm.w;
  p.next_eps = n.norm.eps;
  p.h = n.h;
  p.ld_h = n.ld_h;
  p.h_bf16 = n.h_kind == PI_BF16;
  pi_prof_scope prof(ctx, PI_PROF_OTHER);
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(n.rows * cs), dim3(kThreads), smem_of(p), cs, p));
  return PI_OK;
}
