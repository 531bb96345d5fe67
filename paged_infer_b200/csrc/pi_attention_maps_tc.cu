// Multi-map windowed attention over a bf16 KV pool on the tensor cores (mma.sync; see pi_attention_maps.cu for the
// mathematics).  Scores (in the log2 domain, the distance bias with them) and weights are f32; the weights enter the product with V as two bf16 planes (16 bits).
//
// maps_decode_kernel: one row alone.  CTA = (row, kv head, group of heads, KV split).  The MMA's 16 rows are 16 heads, or
//   8 heads x 2 maps: with two maps the query operand is block diagonal - rows 0-7 hold map 1 in the first half of the
//   key channels and zero in the second, rows 8-15 the other way round - so one product over the concatenated channels
//   scores both maps, and one product with V serves both.  Each warp streams 16-key tiles through a private ring of
//   asynchronous copies; warps merge by log-sum-exp in shared memory, splits through the distributed shared memory of their
//   cluster.
// maps_tile_kernel: portions.  CTA = (sequence, kv head, tile of (token, head) rows); a warp owns 16 rows of one map, the
//   pair of warps with the two maps of the same rows meets in shared memory at the end.  64-key tiles, double buffered.
#include <cooperative_groups.h>
#include <math.h>

#include <algorithm>
#include <type_traits>

#include "pi_attention_maps.cuh"
#include "pi_mma.cuh"

namespace cg = cooperative_groups;

namespace {
using namespace pi_mma;

constexpr float kLog2e = 1.4426950408889634f;

struct TcParams {
  MapsParams m;
  const int32_t* rows;              // decode: the rows that stand alone
  const int32_t *portions, *seq_row0, *seq_n, *seq_start;
  int group, ngroups, nsplit;       // heads per kv head; decode: groups of them per MMA, KV splits
  int out_bf16;
};

__device__ __forceinline__ void store_out(const TcParams& p, size_t i, float v) {
  if (p.out_bf16) static_cast<__nv_bfloat16*>(p.m.out)[i] = __float2bfloat16_rn(v);
  else static_cast<float*>(p.m.out)[i] = v;
}

// Address of key t's row in the pool (K part; V follows the block's keys).
struct Paged {
  const __nv_bfloat16* base;
  const int32_t* table;
  int block_size, kv_heads, head, kw, vp;
  __device__ __forceinline__ const __nv_bfloat16* tile(int lb) const {
    return base + ((size_t)table[lb] * kv_heads + head) * ((size_t)block_size * (kw + vp));
  }
};

// 16 rows of K or V that may lie in several blocks (block sizes that are no multiple of 16): every piece finds its own block.
// Kept out of line: the kernels are short enough for instruction fetch to count.
__device__ __noinline__ void fetch_rows(Paged pg, __nv_bfloat16* dst, int pitch, int t0, int hi, int lane, bool is_v) {
  const int width = is_v ? pg.vp : pg.kw, pr = width / 8;
  for (int c = lane; c < 16 * pr; c += 32) {
    const int r = c / pr, x = (c - r * pr) * 8, t = t0 + r;
    const bool ok = t < hi;
    const __nv_bfloat16* src = pg.base;
    if (ok) {
      const int off = t % pg.block_size;
      src = pg.tile(t / pg.block_size) + (is_v ? (size_t)pg.block_size * pg.kw : (size_t)0) + (size_t)off * width + x;
    }
    cp_async16(smem_addr(dst + r * pitch + x), src, ok ? 16 : 0);
  }
}

// Online softmax step of one accumulator row: running maximum, factor for what is already summed.
__device__ __forceinline__ float new_max(float m, float s_max, float& keep) {
  const float n = fmaxf(m, s_max);
  keep = n == -INFINITY ? 1.f : exp2f(m - n);
  return n;
}

// Weight of a key that weighs by itself: sigmoid of a score in the log2 domain (0 for one of minus infinity).
__device__ __forceinline__ float self_weight(float s) { return __fdividef(1.f, 1.f + exp2f(-s)); }

constexpr int kDecWarps = 4, kDecStages = 3, kMaxSplits = 8;   // splits: a portable cluster

// SELF: sigmoid weights, which need neither maximum nor sum - the merges then just add.
template <int MAPS, int KMAX, int VMAX, bool SELF = false>
__global__ void __launch_bounds__(kDecWarps * 32) maps_decode_kernel(const TcParams p) {
  constexpr int QR = MAPS == 2 ? 2 : 4;     // query registers per 16 channels
  constexpr int HR = 16 / MAPS;             // heads per MMA
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const MapsParams& a = p.m;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = blockIdx.z / p.ngroups, grp = blockIdx.z % p.ngroups, split_i = blockIdx.x;
  const int row = p.rows[blockIdx.y], seq = a.row_seq[row], pos = a.row_pos[row];
  const int kw = MAPS * a.dp, ks_map = a.dp / 16, nks = MAPS * ks_map, nv = a.vp / 8;
  const int kpitch = kw + 8, vpitch = a.vp + 8;
  const int stage_elems = 16 * (kpitch + vpitch);
  __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(smem_raw) + (size_t)warp * kDecStages * stage_elems;
  const Paged pg = {static_cast<const __nv_bfloat16*>(a.base), a.tables + (size_t)seq * a.max_blocks, a.block_size, a.kv_heads, g, kw, a.vp};

  // keys of this CTA: [k_lo, k_hi), tiles start on multiples of 16
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0, hi = min(pos + 1, a.lens[seq] * a.block_size);
  const int t_first = lo / 16, n_tiles = (hi + 15) / 16 - t_first, per = (n_tiles + p.nsplit - 1) / p.nsplit;
  const int tile_end = min(t_first + n_tiles, t_first + (split_i + 1) * per);
  const int tile0 = t_first + split_i * per + warp;
  const bool one_block = a.block_size % 16 == 0;

  const int kpr = kw / 8, vpr = a.vp / 8;               // 16-byte pieces per row
  // physical block of a tile that lies in one block; loaded one tile ahead of its use
  auto block_of = [&](int tile) { return one_block && tile < tile_end ? pg.table[tile * 16 / a.block_size] : 0; };
  auto fetch = [&](int tile, int stage, int pb) {
    __nv_bfloat16* ks = ring + (size_t)stage * stage_elems;
    __nv_bfloat16* vs = ks + 16 * kpitch;
    const int t0 = tile * 16;
    if (one_block) {                                    // 16 rows of K in a piece, 16 rows of V in a piece
      const int off = t0 % a.block_size;
      const __nv_bfloat16* kb = pg.base + ((size_t)pb * a.kv_heads + g) * ((size_t)a.block_size * (kw + a.vp));
      const __nv_bfloat16* vb = kb + (size_t)a.block_size * kw + (size_t)off * a.vp;
      kb += (size_t)off * kw;
      auto copy = [&](__nv_bfloat16* dst, int pitch, int pr, const __nv_bfloat16* src) {
        int r = lane / pr, x = lane - r * pr;
        const int dr = 32 / pr, dx = 32 - dr * pr;
#pragma unroll 4
        for (int c = lane; c < 16 * pr; c += 32) {
          cp_async16(smem_addr(dst + r * pitch + x * 8), src + (size_t)c * 8, t0 + r < hi ? 16 : 0);
          r += dr;
          x += dx;
          if (x >= pr) {
            x -= pr;
            ++r;
          }
        }
      };
      copy(ks, kpitch, kpr, kb);
      copy(vs, vpitch, vpr, vb);
      return;
    }
    fetch_rows(pg, ks, kpitch, t0, hi, lane, false);
    fetch_rows(pg, vs, vpitch, t0, hi, lane, true);
  };

  int pb[kDecStages];
#pragma unroll
  for (int s = 0; s < kDecStages; ++s) pb[s] = block_of(tile0 + s * kDecWarps);
  // Keys in front of this row's own position were written in earlier steps: their tiles are requested ahead of the dependency
  // wait.  The tile with the row's own key is this step's work.
#pragma unroll 1
  for (int late = 0; late < 2; ++late) {
    if (late) pi_grid_dependency_wait();
#pragma unroll 1
    for (int s = 0; s < kDecStages - 1; ++s) {
      const int tile = tile0 + s * kDecWarps;
      if (tile < tile_end && ((tile + 1) * 16 > pos) == (late != 0)) fetch(tile, s, s == 0 ? pb[0] : pb[1]);
      if (late) cp_async_commit();   // the first group also holds what was requested early
    }
  }
  int pb_next = pb[kDecStages - 1];

  // query operand: row r of the MMA = (map r / HR, head r % HR)
  uint32_t qa[KMAX][QR];
  {
    const int r0 = lane >> 2, c0 = (lane & 3) * 2;
    // all loads first (addresses clamped instead of branches, so that they are in flight together), then the packing
    float v[KMAX][QR][2];
    bool ok[2];
    const float* q[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int head = grp * HR + (r0 + 8 * h) % HR;
      ok[h] = head < p.group;
      q[h] = a.q + (size_t)row * a.stride + (size_t)(g * p.group + min(head, p.group - 1)) * MAPS * a.dim;
    }
#pragma unroll
    for (int ks = 0; ks < KMAX; ++ks) {
      const int map = MAPS == 2 && ks >= ks_map ? 1 : 0, d0 = (ks - map * ks_map) * 16 + c0;
#pragma unroll
      for (int j = 0; j < QR; ++j) {
        const int d = d0 + (QR == 2 ? j : j >> 1) * 8;
        const float* src = q[QR == 2 ? 0 : j & 1] + map * a.dim;
        v[ks][j][0] = src[min(d, a.dim - 1)];
        v[ks][j][1] = src[min(d + 1, a.dim - 1)];
      }
    }
#pragma unroll
    for (int ks = 0; ks < KMAX; ++ks) {
      const int map = MAPS == 2 && ks >= ks_map ? 1 : 0, d0 = (ks - map * ks_map) * 16 + c0;
#pragma unroll
      for (int j = 0; j < QR; ++j) {
        const int d = d0 + (QR == 2 ? j : j >> 1) * 8;
        const bool is = ks < nks && ok[QR == 2 ? 0 : j & 1];
        qa[ks][j] = pack(is && d < a.dim ? v[ks][j][0] : 0.f, is && d + 1 < a.dim ? v[ks][j][1] : 0.f);
      }
    }
  }
  float acc[VMAX / 8][4];
#pragma unroll
  for (int j = 0; j < VMAX / 8; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float sc = a.scale * kLog2e;
  float slope[2] = {0.f, 0.f};
  if (a.slopes) {
#pragma unroll
    for (int h = 0; h < 2; ++h) slope[h] = __ldg(a.slopes + g * p.group + min(grp * HR + ((lane >> 2) + 8 * h) % HR, p.group - 1)) * kLog2e;
  }
  float self[2] = {0.f, 0.f};
  if (SELF) {
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      self[h] = __ldg(a.sigmoid_bias + g * p.group + min(grp * HR + ((lane >> 2) + 8 * h) % HR, p.group - 1)) * kLog2e;
      mx[h] = 0.f;                          // warps and splits merge with factors of 1
      l[h] = 1.f;
    }
  }

  int stage = 0;
  for (int tile = tile0; tile < tile_end; tile += kDecWarps) {
    cp_async_wait<kDecStages - 2>();
    __syncwarp();
    const __nv_bfloat16* ks = ring + (size_t)stage * stage_elems;
    const __nv_bfloat16* vs = ks + 16 * kpitch;
    float s[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) s[j][i] = 0.f;
#pragma unroll
    for (int k = 0; k < KMAX; ++k) {
      if (k < nks) {
        uint32_t b[4];   // keys 0-7: channels 0-7, 8-15; keys 8-15 likewise
        ldsm4(b, smem_addr(ks + (size_t)((lane & 7) + ((lane >> 4) << 3)) * kpitch + k * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          if (MAPS == 2) {
            if (k < ks_map) mma(s[j], qa[k][0], 0u, qa[k][1], 0u, b[2 * j], b[2 * j + 1]);
            else mma(s[j], 0u, qa[k][0], 0u, qa[k][1], b[2 * j], b[2 * j + 1]);
          } else {
            mma(s[j], qa[k][0], qa[k][1], qa[k][QR - 2], qa[k][QR - 1], b[2 * j], b[2 * j + 1]);
          }
        }
      }
    }
    const int key = tile * 16 + (lane & 3) * 2;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = key + 8 * j + (i & 1);
        const float v = SELF ? fmaf(s[j][i], sc, self[i >> 1]) : fmaf(slope[i >> 1], (float)(t - pos), s[j][i] * sc);
        s[j][i] = (t >= lo && t < hi) ? v : -INFINITY;
      }
    uint32_t ph[4], pl[4];
    float keep[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {   // MMA rows lane / 4 and lane / 4 + 8
      float w[4];
      if (SELF) {
        keep[h] = 1.f;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int i = 0; i < 2; ++i) w[2 * j + i] = self_weight(s[j][2 * h + i]);
      } else {
        const float tm = quad_max(fmaxf(fmaxf(s[0][2 * h], s[0][2 * h + 1]), fmaxf(s[1][2 * h], s[1][2 * h + 1])));
        mx[h] = new_max(mx[h], tm, keep[h]);
        const float ref = mx[h] == -INFINITY ? 0.f : mx[h];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int i = 0; i < 2; ++i) w[2 * j + i] = exp2f(s[j][2 * h + i] - ref);
        l[h] = l[h] * keep[h] + ((w[0] + w[1]) + (w[2] + w[3]));
      }
      split(w[0], w[1], ph[h], pl[h]);
      split(w[2], w[3], ph[2 + h], pl[2 + h]);
    }
#pragma unroll
    for (int j = 0; j < VMAX / 8; j += 2) {
      if (j < nv) {
        uint32_t b[4];   // value columns j*8.., keys 0-7 and 8-15; then the next eight columns
        ldsm4_t(b, smem_addr(vs + (size_t)((lane & 7) + ((lane >> 3) & 1) * 8) * vpitch + j * 8 + (lane >> 4) * 8));
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          float* d = acc[j + h];
          if (!SELF) {
            d[0] *= keep[0];
            d[1] *= keep[0];
            d[2] *= keep[1];
            d[3] *= keep[1];
          }
          mma(d, ph[0], ph[1], ph[2], ph[3], b[2 * h], b[2 * h + 1]);
          mma(d, pl[0], pl[1], pl[2], pl[3], b[2 * h], b[2 * h + 1]);
        }
      }
    }
    const int next = tile + (kDecStages - 1) * kDecWarps;
    const int pb_now = pb_next;
    pb_next = block_of(next + kDecWarps);
    if (next < tile_end) fetch(next, (stage + kDecStages - 1) % kDecStages, pb_now);
    cp_async_commit();
    stage = (stage + 1) % kDecStages;
  }
  cp_async_wait<0>();
  l[0] = quad_sum(l[0]);
  l[1] = quad_sum(l[1]);

  // ---- merge the warps -----------------------------------------------------------------------------------------------
  __syncthreads();
  float* wacc = reinterpret_cast<float*>(smem_raw);      // [warps][16][vp + 4]
  const int apitch = a.vp + 4;
  __shared__ float s_m[kDecWarps][16], s_l[kDecWarps][16];
  {
    const int r0 = lane >> 2;
    float* w = wacc + (size_t)warp * 16 * apitch;
#pragma unroll
    for (int j = 0; j < VMAX / 8; ++j)
      if (j < nv) {
        const int c = j * 8 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(w + (size_t)r0 * apitch + c) = make_float2(acc[j][0], acc[j][1]);
        *reinterpret_cast<float2*>(w + (size_t)(r0 + 8) * apitch + c) = make_float2(acc[j][2], acc[j][3]);
      }
    if ((lane & 3) == 0) {
      s_m[warp][r0] = mx[0];
      s_m[warp][r0 + 8] = mx[1];
      s_l[warp][r0] = l[0];
      s_l[warp][r0 + 8] = l[1];
    }
  }
  __syncthreads();
  // the CTA's own result, not yet divided by the sum of weights, replaces warp 0's part
  __shared__ float c_m[16], c_l[16];
  for (int r = warp; r < 16; r += kDecWarps) {
    float f[kDecWarps], M = -INFINITY, L = 0.f;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) M = fmaxf(M, s_m[w][r]);
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) {
      f[w] = s_m[w][r] == -INFINITY ? 0.f : exp2f(s_m[w][r] - M);
      L += s_l[w][r] * f[w];
    }
    for (int e = lane; e < a.vp; e += 32) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < kDecWarps; ++w) o = fmaf(wacc[((size_t)w * 16 + r) * apitch + e], f[w], o);
      wacc[(size_t)r * apitch + e] = o;
    }
    if (lane == 0) {
      c_m[r] = M;
      c_l[r] = L;
    }
  }
  // the splits of a row form a cluster: each of them finishes its share of the heads, adding the splits in rank order
  cg::cluster_group cluster = cg::this_cluster();
  if (p.nsplit > 1) cluster.sync();
  else __syncthreads();
  const int rank = p.nsplit > 1 ? (int)cluster.block_rank() : 0;
  // NS parts are read whether they exist or not (ranks clamped, weights zero), so that the loads are in flight together
  auto finish = [&](auto ns_c) {
    constexpr int NS = decltype(ns_c)::value;
    const float *pm[NS], *pl[NS], *pa[NS];
#pragma unroll
    for (int c = 0; c < NS; ++c) {
      const int cr = min(c, p.nsplit - 1);
      pm[c] = NS > 1 ? cluster.map_shared_rank(c_m, cr) : c_m;
      pl[c] = NS > 1 ? cluster.map_shared_rank(c_l, cr) : c_l;
      pa[c] = NS > 1 ? cluster.map_shared_rank(wacc, cr) : wacc;
    }
    for (int h = warp * p.nsplit + rank; h < HR; h += kDecWarps * p.nsplit) {
      const int head = grp * HR + h;
      if (head >= p.group) continue;
      float f[MAPS][NS], l[MAPS][NS];
#pragma unroll
      for (int m = 0; m < MAPS; ++m)
#pragma unroll
        for (int c = 0; c < NS; ++c) {
          f[m][c] = pm[c][h + m * HR];
          l[m][c] = pl[c][h + m * HR];
        }
      const float sink = a.sinks ? __ldg(a.sinks + g * p.group + head) * kLog2e : -INFINITY;
#pragma unroll
      for (int m = 0; m < MAPS; ++m) {
        float M = sink, L = 0.f;
#pragma unroll
        for (int c = 0; c < NS; ++c) M = fmaxf(M, f[m][c]);
        if (a.sinks) L = exp2f(sink - M);
#pragma unroll
        for (int c = 0; c < NS; ++c) {
          f[m][c] = c >= p.nsplit || f[m][c] == -INFINITY ? 0.f : exp2f(f[m][c] - M);
          L = fmaf(l[m][c], f[m][c], L);
        }
        const float inv = SELF ? 1.f : L > 0.f ? (m == 0 ? 1.f : -a.lambda) / L : 0.f;
#pragma unroll
        for (int c = 0; c < NS; ++c) f[m][c] *= inv;
      }
      float d[VMAX / 32], ss = 0.f;
#pragma unroll
      for (int i = 0; i < VMAX / 32; ++i) {
        const int e = min(lane + 32 * i, a.vdim - 1);
        float x[MAPS][NS];
#pragma unroll
        for (int m = 0; m < MAPS; ++m)
#pragma unroll
          for (int c = 0; c < NS; ++c) x[m][c] = pa[c][(size_t)(h + m * HR) * apitch + e];
        d[i] = 0.f;
#pragma unroll
        for (int m = 0; m < MAPS; ++m)
#pragma unroll
          for (int c = 0; c < NS; ++c) d[i] = fmaf(x[m][c], f[m][c], d[i]);
        if (lane + 32 * i < a.vdim) ss = fmaf(d[i], d[i], ss);
      }
      const float r = MAPS == 2 ? a.out_scale / sqrtf(pi_warp_sum(ss) / (float)a.vdim + a.eps) : 1.f;
      const size_t o0 = (size_t)row * a.out_stride + (size_t)(g * p.group + head) * a.vdim;
#pragma unroll
      for (int i = 0; i < VMAX / 32; ++i)
        if (lane + 32 * i < a.vdim) {
          const size_t at = a.gate_per_head ? (size_t)(g * p.group + head) : (size_t)(g * p.group + head) * a.vdim + lane + 32 * i;
          const float gate = a.gate ? pi_sigmoid(a.gate[(size_t)row * a.gate_stride + at]) : 1.f;
          store_out(p, o0 + lane + 32 * i, d[i] * r * gate);
        }
    }
  };
  if (p.nsplit > 1) finish(std::integral_constant<int, kMaxSplits>());
  else finish(std::integral_constant<int, 1>());
  if (p.nsplit > 1) cluster.sync();   // a peer may still be reading this CTA's part
}

constexpr int kTileWarps = 8, kTileKeys = 64;

template <int MAPS, int KMAP, int VMAX, bool SELF = false>
__global__ void __launch_bounds__(kTileWarps * 32, 1) maps_tile_kernel(const TcParams p) {
  constexpr int RG = kTileWarps / MAPS, R = RG * 16;     // row groups of 16 rows
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const MapsParams& a = p.m;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = p.portions[blockIdx.z], g = blockIdx.y, n = p.seq_n[seq];
  const int per_tile = R / p.group;                      // tokens of a tile
  // the last tiles see the most keys: they start first
  const int tile = (int)gridDim.x - 1 - (int)blockIdx.x, tok0 = tile * per_tile;
  if (tok0 >= n) {
    pi_grid_dependency_wait();
    return;
  }
  const int row0 = p.seq_row0[seq], start = p.seq_start[seq], n_tok = min(per_tile, n - tok0);
  const int map = warp / RG, rg = warp % RG;
  const int kw = MAPS * a.dp, nks = a.dp / 16, nv = a.vp / 8, kpitch = kw + 8, vpitch = a.vp + 8;
  const int stage_elems = kTileKeys * (kpitch + vpitch);
  __nv_bfloat16* sm = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  const Paged pg = {static_cast<const __nv_bfloat16*>(a.base), a.tables + (size_t)seq * a.max_blocks, a.block_size, a.kv_heads, g, kw, a.vp};
  const int p_first = start + tok0, p_last = p_first + n_tok - 1;
  const int lo = (a.window > 0 ? max(0, p_first - a.window + 1) : 0) & ~15, hi = min(p_last + 1, a.lens[seq] * a.block_size);
  const int n_blocks = hi > lo ? (hi - lo + kTileKeys - 1) / kTileKeys : 0;

  auto fetch = [&](int kb, int stage) {
    __nv_bfloat16* ks = sm + (size_t)stage * stage_elems;
    __nv_bfloat16* vs = ks + kTileKeys * kpitch;
    const int t0 = lo + kb * kTileKeys;
    // four threads per key: one table lookup serves all chunks of the row
    const int r = tid >> 2, t = t0 + r;
    const bool ok = t < hi;
    const __nv_bfloat16* b = pg.base;
    int off = 0;
    if (ok) {
      const int lb = t / a.block_size;
      b = pg.tile(lb);
      off = t - lb * a.block_size;
    }
    for (int x = (tid & 3) * 8; x < kw; x += 32)
      cp_async16(smem_addr(ks + r * kpitch + x), ok ? (const void*)(b + (size_t)off * kw + x) : a.base, ok ? 16 : 0);
    for (int x = (tid & 3) * 8; x < a.vp; x += 32)
      cp_async16(smem_addr(vs + r * vpitch + x), ok ? (const void*)(b + (size_t)a.block_size * kw + (size_t)off * a.vp + x) : a.base, ok ? 16 : 0);
  };

  pi_grid_dependency_wait();
  if (n_blocks > 0) fetch(0, 0);
  cp_async_commit();

  // this thread's two rows: lane / 4 and lane / 4 + 8 of the row group
  int tpos[2];
  uint32_t qa[KMAP][4];
  {
    const float* q[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = rg * 16 + (lane >> 2) + 8 * h, tok = r / p.group, head = r - tok * p.group;
      const bool ok = tok < n_tok;
      tpos[h] = ok ? p_first + tok : -1;      // -1: sees nothing
      q[h] = a.q + (size_t)(row0 + tok0 + (ok ? tok : 0)) * a.stride + ((size_t)(g * p.group + head) * MAPS + map) * a.dim;
    }
    constexpr int B = KMAP <= 8 ? KMAP : 4;   // of a batch of k steps all loads first, addresses clamped instead of branches
#pragma unroll
    for (int k0 = 0; k0 < KMAP; k0 += B) {
      float v[B][4][2];
#pragma unroll
      for (int ks = 0; ks < B; ++ks)
#pragma unroll
        for (int j = 0; j < 4; ++j) {         // a0: row, a1: row + 8, a2 / a3: channels + 8
          const int d = (k0 + ks) * 16 + (lane & 3) * 2 + (j >> 1) * 8;
          v[ks][j][0] = q[j & 1][min(d, a.dim - 1)];
          v[ks][j][1] = q[j & 1][min(d + 1, a.dim - 1)];
        }
#pragma unroll
      for (int ks = 0; ks < B; ++ks)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int d = (k0 + ks) * 16 + (lane & 3) * 2 + (j >> 1) * 8;
          const bool is = k0 + ks < nks && tpos[j & 1] >= 0;
          qa[k0 + ks][j] = pack(is && d < a.dim ? v[ks][j][0] : 0.f, is && d + 1 < a.dim ? v[ks][j][1] : 0.f);
        }
    }
  }
  float acc[VMAX / 8][4];
#pragma unroll
  for (int j = 0; j < VMAX / 8; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float sc = a.scale * kLog2e;
  float slope[2], sink[2], self[2] = {0.f, 0.f};
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int head = g * p.group + (rg * 16 + (lane >> 2) + 8 * h) % p.group;
    slope[h] = a.slopes ? __ldg(a.slopes + head) * kLog2e : 0.f;
    sink[h] = a.sinks ? __ldg(a.sinks + head) * kLog2e : -INFINITY;
    if (SELF) self[h] = __ldg(a.sigmoid_bias + head) * kLog2e;
  }
  const int win = a.window > 0 ? a.window : 0x3fffffff;

  for (int kb = 0; kb < n_blocks; ++kb) {
    cp_async_wait<0>();
    __syncthreads();                          // this block has landed, the other stage is free
    if (kb + 1 < n_blocks) fetch(kb + 1, (kb + 1) & 1);
    cp_async_commit();
    const __nv_bfloat16* ks = sm + (size_t)(kb & 1) * stage_elems;
    const __nv_bfloat16* vs = ks + kTileKeys * kpitch;
    float s[kTileKeys / 8][4];
#pragma unroll
    for (int j = 0; j < kTileKeys / 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) s[j][i] = 0.f;
#pragma unroll
    for (int k = 0; k < KMAP; ++k)
      if (k < nks) {
#pragma unroll
        for (int j = 0; j < kTileKeys / 8; j += 2) {
          uint32_t b[4];
          ldsm4(b, smem_addr(ks + (size_t)(j * 8 + (lane & 7) + ((lane >> 4) << 3)) * kpitch + map * a.dp + k * 16 + ((lane >> 3) & 1) * 8));
          mma(s[j], qa[k][0], qa[k][1], qa[k][2], qa[k][3], b[0], b[1]);
          mma(s[j + 1], qa[k][0], qa[k][1], qa[k][2], qa[k][3], b[2], b[3]);
        }
      }
    const int t0 = lo + kb * kTileKeys;
    const bool inside = n_tok == per_tile && t0 + kTileKeys - 1 <= p_first && t0 > p_last - win && R == per_tile * p.group;
    float keep[2] = {1.f, 1.f}, ref[2] = {0.f, 0.f};
    if (SELF) {
#pragma unroll
      for (int j = 0; j < kTileKeys / 8; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int t = t0 + j * 8 + (lane & 3) * 2 + (i & 1), q = tpos[i >> 1];
          s[j][i] = (inside || (t <= q && t > q - win && t < hi)) ? self_weight(fmaf(s[j][i], sc, self[i >> 1])) : 0.f;
        }
    } else {
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        float tm = -INFINITY;
#pragma unroll
        for (int j = 0; j < kTileKeys / 8; ++j)
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int t = t0 + j * 8 + (lane & 3) * 2 + i;
            float& v = s[j][2 * h + i];
            v = (inside || (t <= tpos[h] && t > tpos[h] - win && t < hi)) ? fmaf(slope[h], (float)(t - tpos[h]), v * sc) : -INFINITY;
            tm = fmaxf(tm, v);
          }
        mx[h] = new_max(mx[h], quad_max(tm), keep[h]);
        ref[h] = mx[h] == -INFINITY ? 0.f : mx[h];
        l[h] *= keep[h];
      }
    }
    if (!SELF && __any_sync(0xffffffffu, keep[0] != 1.f || keep[1] != 1.f)) {
#pragma unroll
      for (int j = 0; j < VMAX / 8; ++j) {
        acc[j][0] *= keep[0];
        acc[j][1] *= keep[0];
        acc[j][2] *= keep[1];
        acc[j][3] *= keep[1];
      }
    }
#pragma unroll
    for (int c = 0; c < kTileKeys / 16; ++c) {
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const float s0 = s[2 * c + j][2 * h], s1 = s[2 * c + j][2 * h + 1];
          const float w0 = SELF ? s0 : exp2f(s0 - ref[h]), w1 = SELF ? s1 : exp2f(s1 - ref[h]);
          if (!SELF) l[h] += w0 + w1;
          split(w0, w1, ph[2 * j + h], pl[2 * j + h]);
        }
#pragma unroll
      for (int j = 0; j < VMAX / 8; j += 2)
        if (j < nv) {
          uint32_t b[4];
          ldsm4_t(b, smem_addr(vs + (size_t)(c * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vpitch + j * 8 + (lane >> 4) * 8));
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            mma(acc[j + h], ph[0], ph[1], ph[2], ph[3], b[2 * h], b[2 * h + 1]);
            mma(acc[j + h], pl[0], pl[1], pl[2], pl[3], b[2 * h], b[2 * h + 1]);
          }
        }
    }
  }
  cp_async_wait<0>();
  float inv[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const float M = fmaxf(mx[h], sink[h]), f = mx[h] == -INFINITY ? 0.f : exp2f(mx[h] - M);   // the sink joins in
    const float t = quad_sum(l[h]) * f + (a.sinks ? exp2f(sink[h] - M) : 0.f);
    inv[h] = SELF ? 1.f : t > 0.f ? f / t : 0.f;
  }
  float ss[2] = {0.f, 0.f};
  const int apitch = a.vp + 8, r0 = rg * 16 + (lane >> 2);
  float* other = reinterpret_cast<float*>(smem_raw);     // [R][vp + 8]: the second map's rows
  if (MAPS == 2) {
    __syncthreads();
    if (map == 1) {
#pragma unroll
      for (int j = 0; j < VMAX / 8; ++j)
        if (j < nv) {
          const int c = j * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(other + (size_t)r0 * apitch + c) = make_float2(acc[j][0] * inv[0], acc[j][1] * inv[0]);
          *reinterpret_cast<float2*>(other + (size_t)(r0 + 8) * apitch + c) = make_float2(acc[j][2] * inv[1], acc[j][3] * inv[1]);
        }
    }
    __syncthreads();
    if (map == 1) return;
  }
#pragma unroll
  for (int j = 0; j < VMAX / 8; ++j)
    if (j < nv) {
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          float& v = acc[j][2 * h + i];
          v *= inv[h];
          if (MAPS == 2) v -= a.lambda * other[(size_t)(r0 + 8 * h) * apitch + j * 8 + (lane & 3) * 2 + i];
          ss[h] = fmaf(v, v, ss[h]);
        }
    }
  float hg[2] = {1.f, 1.f};
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const float r = MAPS == 2 ? a.out_scale / sqrtf(quad_sum(ss[h]) / (float)a.vdim + a.eps) : 1.f;
    const int rr = r0 + 8 * h, tok = rr / p.group, head = rr - tok * p.group;
    if (tpos[h] < 0) continue;
    if (a.gate && a.gate_per_head) hg[h] = pi_sigmoid(a.gate[(size_t)(row0 + tok0 + tok) * a.gate_stride + g * p.group + head]);
    const size_t o0 = (size_t)(row0 + tok0 + tok) * a.out_stride + (size_t)(g * p.group + head) * a.vdim;
#pragma unroll
    for (int j = 0; j < VMAX / 8; ++j)
      if (j < nv) {
        const int c = j * 8 + (lane & 3) * 2;
        float v0 = acc[j][2 * h] * r, v1 = acc[j][2 * h + 1] * r;
        if (a.gate) {
          const float* gate = a.gate + (size_t)(row0 + tok0 + tok) * a.gate_stride;
          if (a.gate_per_head) {
            v0 *= hg[h];
            v1 *= hg[h];
          } else {
            gate += (size_t)(g * p.group + head) * a.vdim;
            v0 *= pi_sigmoid(gate[min(c, a.vdim - 1)]);
            v1 *= pi_sigmoid(gate[min(c + 1, a.vdim - 1)]);
          }
        }
        if (p.out_bf16 && c + 1 < a.vdim && ((o0 + c) & 1) == 0) {
          *reinterpret_cast<uint32_t*>(static_cast<__nv_bfloat16*>(a.out) + o0 + c) = pack(v0, v1);
        } else {
          if (c < a.vdim) store_out(p, o0 + c, v0);
          if (c + 1 < a.vdim) store_out(p, o0 + c + 1, v1);
        }
      }
  }
}

size_t decode_smem(const MapsParams& a) {
  const size_t ring = (size_t)kDecWarps * kDecStages * 16 * (a.maps * a.dp + 8 + a.vp + 8) * 2;
  return std::max(ring, (size_t)kDecWarps * 16 * (a.vp + 4) * sizeof(float));
}
size_t tile_smem(const MapsParams& a) {
  const size_t stages = (size_t)2 * kTileKeys * (a.maps * a.dp + 8 + a.vp + 8) * 2;
  return std::max(stages, a.maps == 2 ? (size_t)(kTileWarps / 2) * 16 * (a.vp + 8) * sizeof(float) : (size_t)0);
}

typedef void (*TcKernel)(const TcParams);

template <int MAPS, int VMAX, bool SELF>
TcKernel pick_decode(int k) {
  return k <= 8 ? maps_decode_kernel<MAPS, 8, VMAX, SELF> : maps_decode_kernel<MAPS, 16, VMAX, SELF>;
}
template <int MAPS, bool SELF = false>
TcKernel pick_decode(int k, int vp) {
  return vp <= 64 ? pick_decode<MAPS, 64, SELF>(k) : vp <= 128 ? pick_decode<MAPS, 128, SELF>(k) : pick_decode<MAPS, 256, SELF>(k);
}
template <int MAPS, int VMAX, bool SELF>
TcKernel pick_tile(int k) {
  if constexpr (MAPS == 1)   // one map may have wider keys
    if (k > 8) return k <= 12 ? maps_tile_kernel<1, 12, VMAX, SELF> : maps_tile_kernel<1, 16, VMAX, SELF>;
  return k <= 4 ? maps_tile_kernel<MAPS, 4, VMAX, SELF> : maps_tile_kernel<MAPS, 8, VMAX, SELF>;
}
template <int MAPS, bool SELF = false>
TcKernel pick_tile(int k, int vp) {
  return vp <= 64 ? pick_tile<MAPS, 64, SELF>(k) : vp <= 128 ? pick_tile<MAPS, 128, SELF>(k) : pick_tile<MAPS, 256, SELF>(k);
}

// The shared-memory limit of a kernel is raised once per device.
cudaError_t grant(pi_ctx* ctx, TcKernel k, size_t smem) {
  static std::vector<std::pair<TcKernel, pi_smem_grant>> granted;
  for (auto& g : granted)
    if (g.first == k) {
      if (g.second.of(ctx) >= smem) return cudaSuccess;
      g.second.of(ctx) = smem;
      return cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    }
  granted.push_back({k, pi_smem_grant()});
  granted.back().second.of(ctx) = smem;
  return smem > kSmemFree ? cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : cudaSuccess;
}

}  // namespace

bool pi_maps_attention_tc_usable(const pi_ctx* ctx, const pi_maps_attention& a, const pi_kv_view& kv) {
  return ctx->opt_tensor_gemm && kv.kind == PI_BF16 && kv.dp <= (a.maps == 1 ? 256 : 128) && kv.vp <= 256 && a.heads / a.kv_heads <= 16 * kTileWarps / a.maps;
}

pi_status pi_launch_maps_attention_tc(pi_ctx* ctx, const MapsParams& a, int out_kind, const pi_seq_batch& b) {
  TcParams p = {};
  p.m = a;
  p.out_bf16 = out_kind == PI_BF16;
  p.group = a.heads / a.kv_heads;
  p.rows = b.single_rows;
  p.portions = b.portions;
  p.seq_row0 = b.seq_row0;
  p.seq_n = b.seq_n;
  p.seq_start = b.seq_start;
  if (b.n_portions > 0) {
    const int per_tile = 16 * kTileWarps / a.maps / p.group, tiles = (b.max_portion + per_tile - 1) / per_tile;
    const TcKernel k = a.maps == 2 ? pick_tile<2>(a.dp / 16, a.vp) : a.sigmoid_bias ? pick_tile<1, true>(a.dp / 16, a.vp) : pick_tile<1>(a.dp / 16, a.vp);
    const size_t smem = tile_smem(a);
    PI_CUDA(ctx, grant(ctx, k, smem));
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(tiles, a.kv_heads, b.n_portions), dim3(kTileWarps * 32), smem, 1, p));
  }
  if (b.n_single > 0) {
    const int hr = 16 / a.maps;
    p.ngroups = (p.group + hr - 1) / hr;
    // KV splits: one round of CTAs over the GPU, at least one 16-key tile per warp
    const TcKernel k = a.maps == 2 ? pick_decode<2>(2 * a.dp / 16, a.vp) : a.sigmoid_bias ? pick_decode<1, true>(a.dp / 16, a.vp) : pick_decode<1>(a.dp / 16, a.vp);
    const size_t smem = decode_smem(a);
    PI_CUDA(ctx, grant(ctx, k, smem));
    const int keys = a.window > 0 ? std::min(a.window, b.max_pos + 1) : b.max_pos + 1;
    const long ctas = (long)b.n_single * a.kv_heads * p.ngroups, resident = ctx->sm_count * std::max(1L, (long)(ctx->smem_optin / (smem + 2048)));
    p.nsplit = (int)std::max(1L, std::min({resident / ctas, (long)keys / (16 * kDecWarps), (long)kMaxSplits}));
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(p.nsplit, b.n_single, a.kv_heads * p.ngroups), dim3(kDecWarps * 32), smem, p.nsplit, p));
  }
  return PI_OK;
}
