// Routing of tokens to experts.
//
// moe_route_kernel: a warp per token.  Scores s = sigmoid(logit), or the softmax of all logits, or the logits themselves (the weights
// are then the softmax over the chosen alone); choice scores s + correction; the
// experts form equal groups of neighbours, a group's score is its best choice score or the sum of its two best, and only the
// experts of the best groups can be chosen; among them the best choice scores win, ties to the lower index.  Weights: the
// chosen scores s, over their sum if they are brought to sum 1, times a constant.
// moe_lists_kernel: one CTA sorts the (token, choice) pairs by expert - a histogram, its prefix sum, a place for every pair -
// and cuts the experts' rows into column tiles for the grouped GEMM.  (The order of the pairs inside an expert does not
// matter: every row is computed alike wherever it lies.)
// moe_gather_kernel: the activation rows in that order.
#include <algorithm>

#include "pi_layered.cuh"

namespace {

constexpr int kRouteWarps = 8;
constexpr int kListThreads = 1024;

struct RouteParams {
  const float* logits;
  size_t stride;
  const float *bias, *correction;
  int rows, experts, groups, keep, top, score, group_best, renorm;
  float scale;
  int32_t* ids;
  float* weights;
};

struct Best {
  float v;
  int i;
};
// The largest value of the warp, ties to the lower index.  Bits of a float, turned so that their order as an integer is its own.
__device__ __forceinline__ Best warp_best(Best b) {
  const uint32_t bits = __float_as_uint(b.v), key = bits & 0x80000000u ? ~bits : bits | 0x80000000u, top = __reduce_max_sync(0xffffffffu, key);
  return {b.v, (int)__reduce_min_sync(0xffffffffu, key == top ? (uint32_t)b.i : 0x7fffffffu)};
}

__global__ void __launch_bounds__(kRouteWarps * 32) moe_route_kernel(const RouteParams p) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x * kRouteWarps + warp;
  float* choice = sm + (size_t)warp * (2 * p.experts + p.groups);   // [experts], scores [experts], groups [groups]
  float* score = choice + p.experts;
  float* group = score + p.experts;
  pi_grid_dependency_wait();
  if (row >= p.rows) return;
  const float* z = p.logits + (size_t)row * p.stride;
  float top_z = -INFINITY, z_sum = 0.f;
  auto logit = [&](int e) { return z[e] + (p.bias ? __ldg(p.bias + e) : 0.f); };
  if (p.score == PI_SCORE_SOFTMAX) {
    for (int e = lane; e < p.experts; e += 32) top_z = fmaxf(top_z, logit(e));
    top_z = pi_warp_max(top_z);
    for (int e = lane; e < p.experts; e += 32) z_sum += expf(logit(e) - top_z);
    z_sum = pi_warp_sum(z_sum);
  }
  for (int e = lane; e < p.experts; e += 32) {
    const float s = p.score == PI_SCORE_CHOSEN ? logit(e) : p.score == PI_SCORE_SOFTMAX ? expf(logit(e) - top_z) / z_sum : pi_sigmoid(logit(e));
    score[e] = s;
    choice[e] = s + (p.correction ? __ldg(p.correction + e) : 0.f);
  }
  __syncwarp();
  const int n = p.experts / p.groups;
  if (p.keep < p.groups) {
    for (int g = lane; g < p.groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;
      for (int i = 0; i < n; ++i) {
        const float c = choice[g * n + i];
        if (c > a) {
          b = a;
          a = c;
        } else if (c > b) {
          b = c;
        }
      }
      group[g] = n > 1 && p.group_best > 1 ? a + b : a;
    }
    __syncwarp();
    for (int k = 0; k < p.keep; ++k) {                 // a kept group is marked by NaN
      Best b = {-INFINITY, 0x7fffffff};
      for (int g = lane; g < p.groups; g += 32)
        if (group[g] > b.v || (group[g] == b.v && g < b.i)) b = {group[g], g};
      b = warp_best(b);
      if (lane == 0 && b.i < p.groups) group[b.i] = NAN;
      __syncwarp();
    }
    for (int e = lane; e < p.experts; e += 32)
      if (!isnan(group[e / n])) choice[e] = -INFINITY;
    __syncwarp();
  }
  float sum = 0.f, first = -INFINITY;
  int mine[2] = {0, 0};                                // choices lane and lane + 32
  for (int k = 0; k < p.top; ++k) {
    Best b = {-INFINITY, 0x7fffffff};
    for (int e = lane; e < p.experts; e += 32)
      if (choice[e] > b.v || (choice[e] == b.v && choice[e] > -INFINITY && e < b.i)) b = {choice[e], e};
    b = warp_best(b);
    const int e = min(b.i, p.experts - 1);             // (a row of NaN chooses something valid)
    if (lane == (k & 31)) mine[k >> 5] = e;
    first = fmaxf(first, score[e]);
    sum += score[e];
    if (lane == 0) choice[e] = -INFINITY;
    __syncwarp();
  }
  if (p.score == PI_SCORE_CHOSEN) {
    sum = 0.f;
#pragma unroll
    for (int j = 0; j < 2; ++j)
      if (lane + 32 * j < p.top) sum += expf(score[mine[j]] - first);
    sum = pi_warp_sum(sum);
#pragma unroll
    for (int j = 0; j < 2; ++j)
      if (lane + 32 * j < p.top) {
        p.ids[(size_t)row * p.top + lane + 32 * j] = mine[j];
        p.weights[(size_t)row * p.top + lane + 32 * j] = p.scale * expf(score[mine[j]] - first) / sum;
      }
    return;
  }
#pragma unroll
  for (int j = 0; j < 2; ++j)
    if (lane + 32 * j < p.top) {
      p.ids[(size_t)row * p.top + lane + 32 * j] = mine[j];
      p.weights[(size_t)row * p.top + lane + 32 * j] = p.scale * (p.renorm ? score[mine[j]] / (sum + 1e-20f) : score[mine[j]]);
    }
}

__global__ void __launch_bounds__(kListThreads) moe_lists_kernel(const int32_t* ids, int pairs, int experts, int tile_rows, int32_t* place, int32_t* pair_at,
                                                                 int4* tiles, int32_t* n_tiles) {
  extern __shared__ int cnt[];      // [experts] rows, [experts] next place, [experts] first tile
  int* next = cnt + experts;
  int* tile0 = next + experts;
  const int tid = threadIdx.x;
  for (int e = tid; e < experts; e += kListThreads) cnt[e] = 0;
  __syncthreads();
  pi_grid_dependency_wait();
  for (int i = tid; i < pairs; i += kListThreads) atomicAdd(&cnt[ids[i]], 1);
  __syncthreads();
  if (tid < 32) {                   // prefix sums, 32 experts at a time
    int rows = 0, tl = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
      const int e = e0 + tid, c = e < experts ? cnt[e] : 0, t = (c + tile_rows - 1) / tile_rows;
      int sc = c, st = t;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int pc = __shfl_up_sync(0xffffffffu, sc, o), pt = __shfl_up_sync(0xffffffffu, st, o);
        if (tid >= o) {
          sc += pc;
          st += pt;
        }
      }
      if (e < experts) {
        next[e] = rows + sc - c;
        tile0[e] = tl + st - t;
      }
      rows += __shfl_sync(0xffffffffu, sc, 31);
      tl += __shfl_sync(0xffffffffu, st, 31);
    }
    if (tid == 0) *n_tiles = tl;
  }
  __syncthreads();
  for (int e = tid; e < experts; e += kListThreads) {
    const int r0 = next[e], c = cnt[e];
    for (int j = 0; j * tile_rows < c; ++j) tiles[tile0[e] + j] = make_int4(e, r0 + j * tile_rows, min(tile_rows, c - j * tile_rows), 0);
  }
  __syncthreads();
  for (int i = tid; i < pairs; i += kListThreads) {
    const int at = atomicAdd(&next[ids[i]], 1);
    place[i] = at;
    pair_at[at] = i;
  }
}

// 16 bytes at a time; a row's padding travels along.
__global__ void __launch_bounds__(128) moe_gather_kernel(const uint4* h, size_t ld16, uint4* out, const int32_t* pair_at, int top) {
  pi_grid_dependency_wait();
  const uint4* src = h + (size_t)(pair_at[blockIdx.x] / top) * ld16;
  uint4* dst = out + (size_t)blockIdx.x * ld16;
  for (size_t i = threadIdx.x; i < ld16; i += 128) dst[i] = src[i];
}

}  // namespace

int pi_moe_tile_rows(int rows, const pi_moe& m) {
  const int mean = (rows * m.top + m.experts - 1) / m.experts;
  return mean <= 16 ? 16 : mean <= 32 ? 32 : mean <= 64 ? 64 : mean <= 112 ? 128 : 256;
}
int pi_moe_max_tiles(int rows, const pi_moe& m) {
  const int pairs = rows * m.top;
  return std::min(pairs, pairs / pi_moe_tile_rows(rows, m) + std::min(m.experts, pairs));
}

pi_status pi_launch_moe_route(pi_ctx* ctx, const pi_moe& m, const float* logits, size_t stride, int rows, const pi_moe_lists& l) {
  pi_prof_scope prof(ctx, PI_PROF_OTHER);
  const RouteParams p = {logits, stride, m.bias, m.correction, rows, m.experts, m.groups, m.keep, m.top, m.score, m.group_best,
                         m.renorm, m.scale, l.ids, l.weights};
  const size_t smem = (size_t)kRouteWarps * (2 * m.experts + m.groups) * sizeof(float);
  PI_REQUIRE(ctx, smem <= kSmemFit && m.top <= 64, "%d of %d experts are too many", m.top, m.experts);
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, moe_route_kernel, dim3((rows + kRouteWarps - 1) / kRouteWarps), dim3(kRouteWarps * 32), smem, 1, p));
  return PI_OK;
}

pi_status pi_launch_moe_gather(pi_ctx* ctx, const pi_moe& m, int rows, const pi_moe_lists& l, const __nv_bfloat16* h, size_t ld_h, __nv_bfloat16* out) {
  pi_prof_scope prof(ctx, PI_PROF_OTHER);
  PI_REQUIRE(ctx, ld_h % 8 == 0 && (uintptr_t)h % 16 == 0 && (uintptr_t)out % 16 == 0, "activation rows must start on 16-byte boundaries");
  const int pairs = rows * m.top;
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, moe_lists_kernel, dim3(1), dim3(kListThreads), (size_t)3 * m.experts * sizeof(int), 1, (const int32_t*)l.ids, pairs,
                                  m.experts, pi_moe_tile_rows(rows, m), l.place, l.pair_at, l.tiles, l.n_tiles));
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, moe_gather_kernel, dim3(pairs), dim3(128), 0, 1, reinterpret_cast<const uint4*>(h), ld_h / 8, reinterpret_cast<uint4*>(out),
                                  (const int32_t*)l.pair_at, m.top));
  return PI_OK;
}
