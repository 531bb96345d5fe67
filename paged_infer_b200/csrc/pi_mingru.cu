// minGRU: a gated recurrence of single channels whose gates read only the current token, f32 throughout:
//
//   z = sigmoid(zl + bz),  u = ul + bx,  c = u + 1/2 (u >= 0) or sigmoid(u)
//   S_t = (1 - z) S_(t-1) + z c,   out = S_t silu(g)
//
// mingru_scan_kernel: a thread per channel walks the tokens of a sequence, a batch of loads ahead of the arithmetic; the decode
// kernel, and the one of short portions and the f32 mode.
// mingru_chunk_kernel: long portions.  A step is the map S -> a S + b, and maps compose, so time is cut into segments: the warps of
// the CTAs of a cluster each hold the maps of up to kSegment tokens of 32 channels in registers and publish their composition; what
// enters a segment is then a short fold over the segments before it, the CTAs' own through distributed shared memory.  Every operand
// is read once.  1 - z is formed without cancellation; all factors lie in [0, 1], so no product overflows.
#include <cooperative_groups.h>

#include <algorithm>

#include "pi_layered.cuh"

namespace cg = cooperative_groups;

namespace {

constexpr int kScanThreads = 128, kScanAhead = 8;
constexpr int kWarps = 8, kCluster = 8, kSegment = 16, kSegments = kWarps * kCluster;

struct GruParams {
  pi_mingru r;
  const float* proj;
  size_t stride;
  void* out;
  size_t out_stride;
  const int32_t *seqs, *seq_row0, *seq_n, *seq_start, *slot;
};

// One step as a map: S -> a S + b.
struct GruStep {
  float a, b;
};
__device__ __forceinline__ GruStep gru_step(float zl, float ul) {
  const float e = expf(-fabsf(zl)), inv = 1.0f / (1.0f + e);
  const float z = zl >= 0.f ? inv : e * inv;
  return {zl >= 0.f ? e * inv : inv, z * (ul >= 0.f ? ul + 0.5f : pi_sigmoid(ul))};
}

template <typename O>
__global__ void __launch_bounds__(kScanThreads) mingru_scan_kernel(const GruParams p) {
  const pi_mingru& r = p.r;
  const int seq = p.seqs[blockIdx.y], c = blockIdx.x * kScanThreads + threadIdx.x;
  const int row0 = p.seq_row0[seq], n = p.seq_n[seq];
  const bool is = c < r.width;
  float* st = r.state + (size_t)p.slot[seq] * r.state_stride + r.state_off + c;
  // the state was written by an earlier step: it may be read ahead of the dependency wait
  float S = is && p.seq_start[seq] != 0 ? *st : 0.f;
  const float bz = is ? __ldg(r.z_bias + c) : 0.f, bx = is ? __ldg(r.x_bias + c) : 0.f;
  pi_grid_dependency_wait();
  if (!is) return;
  const float* x = p.proj + (size_t)row0 * p.stride + c;
  O* o = static_cast<O*>(p.out) + (size_t)row0 * p.out_stride + c;
  for (int t0 = 0; t0 < n; t0 += kScanAhead) {
    float z[kScanAhead], u[kScanAhead], g[kScanAhead];
#pragma unroll
    for (int j = 0; j < kScanAhead; ++j) {
      const float* xt = x + (size_t)min(t0 + j, n - 1) * p.stride;
      if (j > 0 && t0 + j >= n) continue;
      z[j] = xt[r.col_z];
      u[j] = xt[r.col_x];
      g[j] = xt[r.col_g];
    }
#pragma unroll
    for (int j = 0; j < kScanAhead; ++j) {
      if (t0 + j >= n) break;
      const GruStep s = gru_step(z[j] + bz, u[j] + bx);
      S = fmaf(s.a, S, s.b);
      o[(size_t)(t0 + j) * p.out_stride] = pi_from_f32<O>(S * g[j] * pi_sigmoid(g[j]));
    }
  }
  *st = S;
}

template <typename O>
__global__ void __launch_bounds__(kWarps * 32) mingru_chunk_kernel(const GruParams p) {
  cg::cluster_group cluster = cg::this_cluster();
  const pi_mingru& r = p.r;
  const int rank = (int)cluster.block_rank(), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int seq = p.seqs[blockIdx.y], c = (blockIdx.x / kCluster) * 32 + lane;
  const int row0 = p.seq_row0[seq], n = p.seq_n[seq];
  const bool is = c < r.width;
  __shared__ GruStep seg[kWarps][32];         // this CTA's segments
  __shared__ GruStep whole[2][32];            // this CTA's composition, by pass parity (read by the cluster)
  float* st = r.state + (size_t)p.slot[seq] * r.state_stride + r.state_off + c;
  float S0 = is && p.seq_start[seq] != 0 ? *st : 0.f;
  const float bz = is ? __ldg(r.z_bias + c) : 0.f, bx = is ? __ldg(r.x_bias + c) : 0.f;
  pi_grid_dependency_wait();
  const float* x = p.proj + (size_t)row0 * p.stride + (is ? c : 0);
  O* o = static_cast<O*>(p.out) + (size_t)row0 * p.out_stride + c;
  int pass = 0;
  for (int base = 0; base < n; ++pass) {
    const int left = n - base, len = min(kSegment, (left + kSegments - 1) / kSegments);   // tokens of a segment
    const int t0 = base + (rank * kWarps + warp) * len;
    GruStep m[kSegment];
    float g[kSegment];
    {
      float z[kSegment], u[kSegment];
#pragma unroll
      for (int j = 0; j < kSegment; ++j) {
        const bool ok = j < len && t0 + j < n;
        const float* xt = x + (size_t)(ok ? t0 + j : 0) * p.stride;
        z[j] = ok ? xt[r.col_z] : 0.f;
        u[j] = ok ? xt[r.col_x] : 0.f;
        g[j] = ok ? xt[r.col_g] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < kSegment; ++j) {
        m[j] = gru_step(z[j] + bz, u[j] + bx);
        if (!(j < len && t0 + j < n)) m[j] = {1.f, 0.f};
      }
    }
    GruStep all = m[0];
#pragma unroll
    for (int j = 1; j < kSegment; ++j) all = {all.a * m[j].a, fmaf(m[j].a, all.b, m[j].b)};
    seg[warp][lane] = all;
    __syncthreads();
    GruStep before = {1.f, 0.f};              // this CTA's segments before this one
#pragma unroll
    for (int w = 0; w < kWarps; ++w)
      if (w < warp) {
        const GruStep s = seg[w][lane];
        before = {before.a * s.a, fmaf(s.a, before.b, s.b)};
      }
    if (warp == kWarps - 1) whole[pass & 1][lane] = {before.a * all.a, fmaf(all.a, before.b, all.b)};
    cluster.sync();
    float S = S0;                             // what enters this CTA, and what leaves the cluster
    GruStep part[kCluster];
#pragma unroll
    for (int k = 0; k < kCluster; ++k) part[k] = *cluster.map_shared_rank(&whole[pass & 1][lane], k);
#pragma unroll
    for (int k = 0; k < kCluster; ++k) {
      if (k == rank) S = S0;
      S0 = fmaf(part[k].a, S0, part[k].b);
    }
    S = fmaf(before.a, S, before.b);
    if (is) {
#pragma unroll
      for (int j = 0; j < kSegment; ++j) {
        if (!(j < len && t0 + j < n)) break;
        S = fmaf(m[j].a, S, m[j].b);
        o[(size_t)(t0 + j) * p.out_stride] = pi_from_f32<O>(S * g[j] * pi_sigmoid(g[j]));
      }
    }
    base += len * kSegments;
  }
  cluster.sync();                             // everybody has read the old state, and nobody reads a peer any more
  if (is && rank == 0 && warp == 0) *st = S0;
}

}  // namespace

pi_status pi_launch_mingru(pi_ctx* ctx, const pi_mingru& r, const float* proj, size_t stride, void* out, size_t out_stride, int out_kind,
                           const pi_seq_batch& b) {
  pi_prof_scope prof(ctx, PI_PROF_RECURRENCE);
  GruParams p = {r, proj, stride, out, out_stride, b.scan_seqs, b.seq_row0, b.seq_n, b.seq_start, b.slot};
  if (b.n_scan > 0) {
    auto k = out_kind == PI_BF16 ? mingru_scan_kernel<__nv_bfloat16> : mingru_scan_kernel<float>;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3((r.width + kScanThreads - 1) / kScanThreads, b.n_scan), dim3(kScanThreads), 0, 1, p));
  }
  if (b.n_chunk_seqs > 0) {
    p.seqs = b.chunk_seqs;
    auto k = out_kind == PI_BF16 ? mingru_chunk_kernel<__nv_bfloat16> : mingru_chunk_kernel<float>;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3((r.width + 31) / 32 * kCluster, b.n_chunk_seqs), dim3(kWarps * 32), 0, kCluster, p));
  }
  return PI_OK;
}
