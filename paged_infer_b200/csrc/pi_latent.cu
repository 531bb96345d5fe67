// Latent attention over the paged pool.  A token's keys and values are linear in one latent vector c (of unit root mean
// square, times a weight) that all heads share; beside it a rotated key part k_r, also shared:
//
//   score_h(t, s) = scale (q_h . (UK_h c_s) + r_h . k_r,s),   a_h = sum of softmax weights (UV_h c_s),   out_h = sigmoid(g_h) a_h
//
// Only c and k_r are cached.  Two ways through, with the same result up to rounding:
//   absorbed    q_h . (UK_h c) = (UK_h^T q_h) . c and sum p (UV_h c) = UV_h (sum p c): queries are taken into latent space, the
//               cached rows serve as keys and (their first channels) as values of every head.  Decoding, short portions, f32.
//                 1. latent_prepare_kernel   cache write (norm, rotation) and UK^T q      2. attention over the latents
//                 3. latent_out_kernel       UV and the output gate
//   expanded    portions of kExpandPortion tokens and more (bf16): the latents of the keys in view are gathered, one GEMM
//               spells out keys and values of all heads into a scratch pool, and the windowed tile kernel of multi-map
//               attention runs on it: a third of the arithmetic per (query, key) pair at a latent of four head sizes.
//
// latent_decode_kernel (bf16 pool, mma.sync): CTA = (row, group of 16 heads = the MMA's rows, KV split).  Tiles of 64 keys, two
// in flight.  A warp scores 16 keys over a quarter of the channels, its queries in registers; the softmax meets in shared
// memory, every warp sums its own value channels over all 64 keys, so that accumulators never merge inside a CTA.  The
// weights enter as two bf16 planes (16 bits).  Splits of a row form a cluster and merge through distributed shared memory.
#include <cooperative_groups.h>
#include <limits.h>
#include <math.h>

#include <algorithm>
#include <type_traits>

#include "pi_attention_maps.cuh"
#include "pi_mma.cuh"

namespace cg = cooperative_groups;

namespace {
using namespace pi_mma;

constexpr float kLog2e = 1.4426950408889634f;

// ---- a matrix per head, applied to a few rows ------------------------------------------------------------------------------
constexpr int kHeadThreads = 128, kHeadCols = 64, kHeadRows = 16;

struct HeadTile {
  __nv_bfloat16 *w, *x;
  int pitch, kp;
};
__device__ __forceinline__ HeadTile head_tile(unsigned char* smem, int K) {
  HeadTile t;
  t.kp = (K + 15) / 16 * 16;
  t.pitch = t.kp + 8;
  t.w = reinterpret_cast<__nv_bfloat16*>(smem);
  t.x = t.w + kHeadCols * t.pitch;
  return t;
}
size_t head_smem(int K) { return (size_t)(kHeadCols + kHeadRows) * ((K + 15) / 16 * 16 + 8) * 2; }

// Request rows n0 .. n0 + 63 of W [N][ld] (zeros outside); waits for nothing.
__device__ __forceinline__ void head_weights(const HeadTile& t, const __nv_bfloat16* W, size_t ld, int N, int n0) {
  const int pieces = t.kp / 8;
  for (int i = threadIdx.x; i < kHeadCols * pieces; i += kHeadThreads) {
    const int n = i / pieces, k = (i - n * pieces) * 8;
    const bool ok = n0 + n < N && k < (int)ld;
    cp_async16(smem_addr(t.w + n * t.pitch + k), ok ? W + (size_t)(n0 + n) * ld + k : W, ok ? 16 : 0);
  }
  cp_async_commit();
}
__device__ __forceinline__ float as_f32(float v) { return v; }
__device__ __forceinline__ float as_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

// 16 rows at a time: x(i) points to the K inputs of row i < rows (f32 or bf16; `vec`: on 16-byte boundaries, K a multiple of 8),
// use(i, n, value).
template <typename X, typename F>
__device__ __forceinline__ void head_rows(const HeadTile& t, int K, int N, int n0, int rows, int z, int nz, bool vec, X&& x, F&& use) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  constexpr bool kF32 = std::is_same<typename std::decay<decltype(*x(0))>::type, float>::value;
  for (int m0 = z * kHeadRows; m0 < rows; m0 += nz * kHeadRows) {
    __syncthreads();     // the last rows have been read
    if (vec) {
      const int pieces = t.kp / 8;
#pragma unroll 4
      for (int i = threadIdx.x; i < kHeadRows * pieces; i += kHeadThreads) {
        const int m = i / pieces, k = (i - m * pieces) * 8;
        const bool ok = m0 + m < rows && k < K;
        const auto* src = x(min(m0 + m, rows - 1)) + min(k, K - 8);
        __nv_bfloat16* dst = t.x + m * t.pitch + k;
        if constexpr (kF32) {
          const float4 a = *reinterpret_cast<const float4*>(src), b = *reinterpret_cast<const float4*>(src + 4);
          *reinterpret_cast<uint4*>(dst) = ok ? make_uint4(pack(a.x, a.y), pack(a.z, a.w), pack(b.x, b.y), pack(b.z, b.w)) : make_uint4(0, 0, 0, 0);
        } else {
          cp_async16(smem_addr(dst), src, ok ? 16 : 0);
        }
      }
      cp_async_commit();
    } else {
      for (int i = threadIdx.x; i < kHeadRows * t.kp; i += kHeadThreads) {
        const int m = i / t.kp, k = i - m * t.kp;
        t.x[m * t.pitch + k] = __float2bfloat16_rn(m0 + m < rows && k < K ? as_f32(x(m0 + m)[k]) : 0.f);
      }
    }
    cp_async_wait<0>();
    __syncthreads();
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 4
    for (int k = 0; k < t.kp; k += 16) {
      uint32_t a[4], b[4];
      ldsm4(a, smem_addr(t.x + ((lane & 7) + ((lane >> 3) & 1) * 8) * t.pitch + k + (lane >> 4) * 8));
      ldsm4(b, smem_addr(t.w + (warp * 16 + (lane & 7) + ((lane >> 4) << 3)) * t.pitch + k + ((lane >> 3) & 1) * 8));
      mma(acc[0], a[0], a[1], a[2], a[3], b[0], b[1]);
      mma(acc[1], a[0], a[1], a[2], a[3], b[2], b[3]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int m = m0 + (lane >> 2) + (i >> 1) * 8, n = n0 + warp * 16 + j * 8 + (lane & 3) * 2 + (i & 1);
        if (m < rows && n < N) use(m, n, acc[j][i]);
      }
  }
}
// The same in f32 on the CUDA cores, one row: xs [K] in shared memory.
template <typename F>
__device__ __forceinline__ void head_row_f32(const uint16_t* W, size_t ld, int N, int K, const float* xs, F&& use) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int n = warp; n < N; n += kHeadThreads / 32) {
    float a = 0.f;
    for (int k = lane; k < K; k += 32) a = fmaf(pi_bf16_bits_to_f32(W[(size_t)n * ld + k]), xs[k], a);
    a = pi_warp_sum(a);
    if (lane == 0) use(n, a);
  }
}

struct LatentParams {
  float* proj;
  size_t stride;
  int heads, dim, rot, vdim, rank, rp, dp, window, block_size, col_q, col_kv, col_g;
  float scale, eps;
  const float *norm, *rope_cos, *rope_sin;
  const void *uk_t, *uv;
  size_t uk_ld, uv_ld;
  void *q, *o, *base, *out;
  size_t out_stride;
  const int32_t *row_seq, *row_pos, *seq_n, *seq_start, *lens, *tables, *latent_rows;
  int max_blocks, rows, n_latent, expand_min;
  int slices, row_splits;      // absorb: 64-channel slices of the latent, CTAs that share the rows of one
  int groups, nsplit;          // decode: groups of 16 heads, KV splits
  int block_shift;             // block_size is 1 << block_shift; -1: it is no power of two
};

// CTA i < rows: row i into the pool, its queries rotated.  The CTAs behind: queries of the latent rows into latent space.
template <typename T>
__global__ void __launch_bounds__(kHeadThreads) latent_prepare_kernel(const LatentParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  constexpr bool kF32 = std::is_same<T, float>::value;
  const int tid = threadIdx.x, qd = p.dim + p.rot, half = p.rot >> 1;
  T* q = static_cast<T*>(p.q);
  if ((int)blockIdx.x >= p.rows) {
    const int i = (int)blockIdx.x - p.rows;
    if (kF32) {
      const int head = i % p.heads, row = p.latent_rows[i / p.heads];
      float* xs = reinterpret_cast<float*>(smem);
      pi_grid_dependency_wait();
      for (int k = tid; k < p.dim; k += kHeadThreads) xs[k] = p.proj[(size_t)row * p.stride + p.col_q + (size_t)head * qd + k];
      __syncthreads();
      T* dst = q + ((size_t)row * p.heads + head) * p.dp;
      head_row_f32(static_cast<const uint16_t*>(p.uk_t) + (size_t)head * p.rank * p.uk_ld, p.uk_ld, p.rank, p.dim, xs,
                   [&](int n, float v) { dst[n] = pi_from_f32<T>(v); });
    } else {
      const int z = i % p.row_splits, s = i / p.row_splits, head = s / p.slices, n0 = (s % p.slices) * kHeadCols;
      const HeadTile t = head_tile(smem, p.dim);
      head_weights(t, static_cast<const __nv_bfloat16*>(p.uk_t) + (size_t)head * p.rank * p.uk_ld, p.uk_ld, p.rank, n0);
      pi_grid_dependency_wait();
      const bool vec = p.dim % 8 == 0 && qd % 4 == 0 && p.stride % 4 == 0 && p.col_q % 4 == 0;
      head_rows(t, p.dim, p.rank, n0, p.n_latent, z, p.row_splits, vec,
                [&](int m) { return p.proj + (size_t)p.latent_rows[m] * p.stride + p.col_q + (size_t)head * qd; },
                [&](int m, int n, float v) { q[((size_t)p.latent_rows[m] * p.heads + head) * p.dp + n] = pi_from_f32<T>(v); });
    }
    return;
  }
  const int row = blockIdx.x, seq = p.row_seq[row], pos = p.row_pos[row], lb = pos / p.block_size, off = pos - lb * p.block_size;
  const int pb = lb < p.lens[seq] ? p.tables[(size_t)seq * p.max_blocks + lb] : -1;
  const bool expanded = p.seq_n[seq] >= p.expand_min;
  const float* cs = p.rope_cos + (size_t)pos * half;
  const float* sn = p.rope_sin + (size_t)pos * half;
  pi_grid_dependency_wait();
  float* x = p.proj + (size_t)row * p.stride;
  const float* c = x + p.col_kv;
  __shared__ float red[kHeadThreads / 32];
  float ss = 0.f;
  for (int i = tid; i < p.rank; i += kHeadThreads) ss = fmaf(c[i], c[i], ss);
  ss = pi_warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = red[0];
#pragma unroll
  for (int w = 1; w < kHeadThreads / 32; ++w) ss += red[w];
  if (pb >= 0) {
    const float inv = 1.0f / sqrtf(ss / (float)p.rank + p.eps);
    T* dst = static_cast<T*>(p.base) + ((size_t)pb * p.block_size + off) * p.dp;
    for (int i = tid; i < p.rank; i += kHeadThreads) dst[i] = pi_from_f32<T>(c[i] * inv * __ldg(p.norm + i));
    for (int j = tid; j < half; j += kHeadThreads) {
      const float u = c[p.rank + 2 * j], v = c[p.rank + 2 * j + 1];
      dst[p.rp + 2 * j] = pi_from_f32<T>(u * cs[j] - v * sn[j]);
      dst[p.rp + 2 * j + 1] = pi_from_f32<T>(v * cs[j] + u * sn[j]);
    }
  }
  for (int i = tid; i < p.heads * half; i += kHeadThreads) {
    const int h = i / half, j = i - h * half;
    float* r = x + p.col_q + (size_t)h * qd + p.dim + 2 * j;
    const float u = r[0], v = r[1], nu = u * cs[j] - v * sn[j], nv = v * cs[j] + u * sn[j];
    if (expanded) {
      r[0] = nu;
      r[1] = nv;
    } else {
      T* dst = q + ((size_t)row * p.heads + h) * p.dp + p.rp + 2 * j;
      dst[0] = pi_from_f32<T>(nu);
      dst[1] = pi_from_f32<T>(nv);
    }
  }
  if (!expanded) {   // what pads the latent and the rotated part
    const int pad0 = p.rp - p.rank, pads = pad0 + p.dp - p.rp - p.rot;
    for (int i = tid; i < p.heads * pads; i += kHeadThreads) {
      const int h = i / pads, j = i - h * pads;
      q[((size_t)row * p.heads + h) * p.dp + (j < pad0 ? p.rank + j : p.rp + p.rot + j - pad0)] = pi_from_f32<T>(0.f);
    }
  }
}

// UV and the output gate for the latent rows.
template <typename O>
__global__ void __launch_bounds__(kHeadThreads) latent_out_kernel(const LatentParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  const int head = blockIdx.y, n0 = blockIdx.x * kHeadCols;
  const HeadTile t = head_tile(smem, p.rank);
  head_weights(t, static_cast<const __nv_bfloat16*>(p.uv) + (size_t)head * p.vdim * p.uv_ld, p.uv_ld, p.vdim, n0);
  pi_grid_dependency_wait();
  const __nv_bfloat16* o = static_cast<const __nv_bfloat16*>(p.o);
  head_rows(t, p.rank, p.vdim, n0, p.n_latent, blockIdx.z, gridDim.z, p.rank % 8 == 0,
            [&](int m) { return o + ((size_t)p.latent_rows[m] * p.heads + head) * p.rank; },
            [&](int m, int n, float v) {
              const size_t row = p.latent_rows[m];
              static_cast<O*>(p.out)[row * p.out_stride + head * p.vdim + n] = pi_from_f32<O>(v * pi_sigmoid(p.proj[row * p.stride + p.col_g + head * p.vdim + n]));
            });
}
template <typename O>
__global__ void __launch_bounds__(kHeadThreads) latent_out_f32_kernel(const LatentParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  float* xs = reinterpret_cast<float*>(smem);
  const int head = blockIdx.x;
  const size_t row = p.latent_rows[blockIdx.y];
  pi_grid_dependency_wait();
  for (int k = threadIdx.x; k < p.rank; k += kHeadThreads) xs[k] = static_cast<const float*>(p.o)[(row * p.heads + head) * p.rank + k];
  __syncthreads();
  head_row_f32(static_cast<const uint16_t*>(p.uv) + (size_t)head * p.vdim * p.uv_ld, p.uv_ld, p.vdim, p.rank, xs, [&](int n, float v) {
    static_cast<O*>(p.out)[row * p.out_stride + head * p.vdim + n] = pi_from_f32<O>(v * pi_sigmoid(p.proj[row * p.stride + p.col_g + head * p.vdim + n]));
  });
}

// ---- decode attention over the latents ---------------------------------------------------------------------------------------
constexpr int kDecWarps = 16, kDecThreads = kDecWarps * 32, kKeys = 64, kStages = 2, kMaxSplits = 16;
constexpr int kSPitch = kKeys + 8, kPPitch = kKeys + 8;

struct DecodeSmem {
  size_t s, p, acc, total;         // byte offsets: scores and weights behind the ring; the finished sums take the ring's place
};
__host__ __device__ inline DecodeSmem decode_smem(int dp, int rp) {
  DecodeSmem s;
  const size_t ring = (size_t)kStages * kKeys * (dp + 8) * 2, acc = (size_t)16 * (rp + 4) * 4;
  s.acc = 0;
  s.s = ring > acc ? ring : acc;
  s.p = s.s + (size_t)4 * 16 * kSPitch * 4;
  s.total = s.p + (size_t)2 * 16 * kPPitch * 2;
  return s;
}

// QMAX: steps of 16 channels per warp (a quarter of a row), UMAX: units of 16 value channels per warp.
template <int QMAX, int UMAX>
__global__ void __launch_bounds__(kDecThreads, 1) latent_decode_kernel(const LatentParams p) {
  static_assert(kStages == 2, "the tile behind the current one is in flight");
  extern __shared__ __align__(16) unsigned char smem[];
  const DecodeSmem lay = decode_smem(p.dp, p.rp);
  __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(smem);
  float* scores = reinterpret_cast<float*>(smem + lay.s);     // [quarter of the channels][16][kSPitch]
  __nv_bfloat16* phi = reinterpret_cast<__nv_bfloat16*>(smem + lay.p);   // weights, two planes [16][kPPitch]
  __nv_bfloat16* plo = phi + 16 * kPPitch;
  __shared__ float s_keep[16], c_m[16], c_l[16];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, split_i = blockIdx.x, h0 = blockIdx.z * 16;
  const int row = p.latent_rows[blockIdx.y], seq = p.row_seq[row], pos = p.row_pos[row], settled = p.seq_start[seq];
  const int32_t* table = p.tables + (size_t)seq * p.max_blocks;
  const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(p.base);
  const int pitch = p.dp + 8, units = p.rp / 16;
  // this warp scores keys 16 (warp % 4).. over its quarter of the channels
  const int quarter = warp >> 2, nks = p.dp / 16, k0 = nks * quarter / 4, n_k = nks * (quarter + 1) / 4 - k0;

  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0, hi = min(pos + 1, p.lens[seq] * p.block_size);
  const int t_first = lo / kKeys, n_tiles = max(0, (hi + kKeys - 1) / kKeys - t_first), per = (n_tiles + p.nsplit - 1) / p.nsplit;
  const int tile0 = t_first + split_i * per, tile_end = min(t_first + n_tiles, tile0 + per);

  // eight threads per key; its physical block is looked up a tile ahead of the request
  const int fr = tid >> 3, fx = (tid & 7) * 8;
  auto logical = [&](int t) { return p.block_shift >= 0 ? t >> p.block_shift : t / p.block_size; };
  auto block_of = [&](int tile) {
    const int t = tile * kKeys + fr;
    return tile < tile_end && t < hi ? table[logical(t)] : -1;
  };
  auto fetch = [&](int tile, int stage, int pb) {
    const int t = tile * kKeys + fr;
    const __nv_bfloat16* src = (pb >= 0 ? base + ((size_t)pb * p.block_size + (t - logical(t) * p.block_size)) * p.dp : base) + fx;
    const uint32_t dst = smem_addr(ring + ((size_t)stage * kKeys + fr) * pitch + fx), bytes = pb >= 0 ? 16 : 0;
#pragma unroll 3
    for (int x = 0; x < p.dp - fx; x += 64) cp_async16(dst + x * 2, src + x, bytes);
  };
  const int pb0 = block_of(tile0), pb1 = block_of(tile0 + 1);
  // tiles of keys that earlier steps wrote are requested ahead of the dependency wait
  const bool early0 = (tile0 + 1) * kKeys <= settled, early1 = (tile0 + 2) * kKeys <= settled;
  if (early0 && tile0 < tile_end) fetch(tile0, 0, pb0);
  if (early0 && early1 && tile0 + 1 < tile_end) fetch(tile0 + 1, 1, pb1);
  pi_grid_dependency_wait();
  if (!early0 && tile0 < tile_end) fetch(tile0, 0, pb0);
  cp_async_commit();                 // the first group also holds what was requested early
  if (!(early0 && early1) && tile0 + 1 < tile_end) fetch(tile0 + 1, 1, pb1);
  cp_async_commit();
  int pb_next = block_of(tile0 + 2);

  uint32_t qa[QMAX][4];
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q) + ((size_t)row * p.heads + h0) * p.dp + (lane & 3) * 2;
    const int r0 = lane >> 2, live = p.heads - h0;
#pragma unroll
    for (int k = 0; k < QMAX; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) {   // a0: head, a1: head + 8, a2 / a3: channels + 8; outside: a valid address and zero
        const int r = r0 + (j & 1) * 8;
        const bool ok = r < live && k < n_k;
        const uint32_t v = *reinterpret_cast<const uint32_t*>(q + (ok ? (size_t)r * p.dp + (k0 + k) * 16 + (j >> 1) * 8 : (size_t)0));
        qa[k][j] = ok ? v : 0u;
      }
  }
  float acc[UMAX][2][4];
#pragma unroll
  for (int u = 0; u < UMAX; ++u)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[u][j][i] = 0.f;
  // softmax: warp = head, lane = two keys
  const int sk = lane * 2;
  float mx = -INFINITY, l = 0.f;
  const float sc = p.scale * kLog2e;
  const int r0 = lane >> 2;

  for (int tile = tile0; tile < tile_end; ++tile) {
    const int stage = (tile - tile0) & 1;
    const __nv_bfloat16* ks = ring + (size_t)stage * kKeys * pitch;
    cp_async_wait<1>();
    __syncthreads();                 // the tile has landed
    {
      float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
      const uint32_t kb = smem_addr(ks + (size_t)((warp & 3) * 16 + (lane & 7) + ((lane >> 4) << 3)) * pitch + k0 * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int k = 0; k < QMAX; ++k) {
        if (k < n_k) {
          uint32_t b[4];             // keys 0-7: channels 0-7, 8-15; keys 8-15 likewise
          ldsm4(b, kb + k * 32);
          mma(s[0], qa[k][0], qa[k][1], qa[k][2], qa[k][3], b[0], b[1]);
          mma(s[1], qa[k][0], qa[k][1], qa[k][2], qa[k][3], b[2], b[3]);
        }
      }
      float* out = scores + (size_t)(quarter * 16 + r0) * kSPitch + (warp & 3) * 16 + (lane & 3) * 2;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        *reinterpret_cast<float2*>(out + j * 8) = make_float2(s[j][0], s[j][1]);
        *reinterpret_cast<float2*>(out + 8 * kSPitch + j * 8) = make_float2(s[j][2], s[j][3]);
      }
    }
    __syncthreads();
    {
      float v[2] = {0.f, 0.f};
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 x = *reinterpret_cast<const float2*>(scores + (size_t)(q * 16 + warp) * kSPitch + sk);
        v[0] += x.x;
        v[1] += x.y;
      }
      const int t = tile * kKeys + sk;
#pragma unroll
      for (int j = 0; j < 2; ++j) v[j] = t + j >= lo && t + j < hi ? v[j] * sc : -INFINITY;
      const float n = fmaxf(mx, pi_warp_max(fmaxf(v[0], v[1])));
      const float keep = n == -INFINITY ? 1.f : exp2f(mx - n), ref = n == -INFINITY ? 0.f : n;
      mx = n;
#pragma unroll
      for (int j = 0; j < 2; ++j) v[j] = exp2f(v[j] - ref);
      l = l * keep + (v[0] + v[1]);
      split(v[0], v[1], *reinterpret_cast<uint32_t*>(phi + warp * kPPitch + sk), *reinterpret_cast<uint32_t*>(plo + warp * kPPitch + sk));
      if (lane == 0) s_keep[warp] = keep;
    }
    __syncthreads();
    const float keep0 = s_keep[r0], keep1 = s_keep[r0 + 8];
    if (__any_sync(0xffffffffu, keep0 != 1.f || keep1 != 1.f)) {
#pragma unroll
      for (int u = 0; u < UMAX; ++u)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          acc[u][j][0] *= keep0;
          acc[u][j][1] *= keep0;
          acc[u][j][2] *= keep1;
          acc[u][j][3] *= keep1;
        }
    }
#pragma unroll
    for (int k = 0; k < kKeys / 16; ++k) {
      uint32_t ph[4], pl[4];
      const int pr = ((lane & 7) + ((lane >> 3) & 1) * 8) * kPPitch + k * 16 + (lane >> 4) * 8;
      ldsm4(ph, smem_addr(phi + pr));
      ldsm4(pl, smem_addr(plo + pr));
      const uint32_t vb = smem_addr(ks + (size_t)(k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (lane >> 4) * 8);
#pragma unroll
      for (int u = 0; u < UMAX; ++u) {
        const int unit = warp + u * kDecWarps;
        if (unit < units) {
          uint32_t b[4];
          ldsm4_t(b, vb + unit * 32);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            mma(acc[u][j], ph[0], ph[1], ph[2], ph[3], b[2 * j], b[2 * j + 1]);
            mma(acc[u][j], pl[0], pl[1], pl[2], pl[3], b[2 * j], b[2 * j + 1]);
          }
        }
      }
    }
    __syncthreads();                 // the stage has been read
    if (tile + 2 < tile_end) fetch(tile + 2, stage, pb_next);
    cp_async_commit();
    pb_next = block_of(tile + 3);
  }
  cp_async_wait<0>();
  __syncthreads();

  // ---- the CTA's sums (not divided yet), then the splits ------------------------------------------------------------------------
  float* wacc = reinterpret_cast<float*>(smem + lay.acc);   // [16][rp + 4]
  const int apitch = p.rp + 4;
#pragma unroll
  for (int u = 0; u < UMAX; ++u) {
    const int unit = warp + u * kDecWarps;
    if (unit < units)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int c = unit * 16 + j * 8 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(wacc + (size_t)r0 * apitch + c) = make_float2(acc[u][j][0], acc[u][j][1]);
        *reinterpret_cast<float2*>(wacc + (size_t)(r0 + 8) * apitch + c) = make_float2(acc[u][j][2], acc[u][j][3]);
      }
  }
  l = pi_warp_sum(l);
  if (lane == 0) {
    c_m[warp] = mx;
    c_l[warp] = l;
  }
  cg::cluster_group cluster = cg::this_cluster();
  if (p.nsplit > 1) cluster.sync();
  else __syncthreads();
  const int rank = p.nsplit > 1 ? (int)cluster.block_rank() : 0;
  // warp = head; channels are dealt to the splits.  NS parts are read whether they exist or not (ranks
  // clamped, weights zero), so that the loads are in flight together.
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
    for (int r = warp; r < min(16, p.heads - h0); r += kDecWarps) {
      float f[NS], ll[NS], M = -INFINITY, L = 0.f;
#pragma unroll
      for (int c = 0; c < NS; ++c) {
        f[c] = pm[c][r];
        ll[c] = pl[c][r];
      }
#pragma unroll
      for (int c = 0; c < NS; ++c) M = fmaxf(M, f[c]);
#pragma unroll
      for (int c = 0; c < NS; ++c) {
        f[c] = c >= p.nsplit || f[c] == -INFINITY ? 0.f : exp2f(f[c] - M);
        L = fmaf(ll[c], f[c], L);
      }
      const float inv = L > 0.f ? 1.f / L : 0.f;
      __nv_bfloat16* o = static_cast<__nv_bfloat16*>(p.o) + ((size_t)row * p.heads + h0 + r) * p.rank;
      for (int e = rank * 32 + lane; e < p.rank; e += p.nsplit * 32) {
        float x[NS], t = 0.f;
#pragma unroll
        for (int c = 0; c < NS; ++c) x[c] = pa[c][(size_t)r * apitch + e];
#pragma unroll
        for (int c = 0; c < NS; ++c) t = fmaf(x[c], f[c], t);
        o[e] = __float2bfloat16_rn(t * inv);
      }
    }
  };
  if (p.nsplit > 8) finish(std::integral_constant<int, kMaxSplits>());
  else if (p.nsplit > 1) finish(std::integral_constant<int, 8>());
  else finish(std::integral_constant<int, 1>());
  if (p.nsplit > 1) cluster.sync();   // a peer may still be reading this CTA's part
}

// ---- expanded portions -------------------------------------------------------------------------------------------------------------
struct GatherParams {
  const __nv_bfloat16* base;
  int dp, rp, rank, rot, block_size;
  const int32_t *key_seq, *key_pos, *exp_lo, *tables;
  int max_blocks;
  const int32_t* exp_tables;
  int exp_max_blocks;
  __nv_bfloat16 *keys, *pool;
  int heads, dim, dpk, vpk;
};

// CTA per key: its latent into a dense row, its rotated part (and zeros behind) into the scratch rows of all heads.
__global__ void __launch_bounds__(128) latent_gather_kernel(const GatherParams p) {
  const int i = blockIdx.x, tid = threadIdx.x, seq = p.key_seq[i], kp = p.key_pos[i], pos = p.exp_lo[seq] + kp;
  const int lb = pos / p.block_size;
  const __nv_bfloat16* src = p.base + ((size_t)p.tables[(size_t)seq * p.max_blocks + lb] * p.block_size + (pos - lb * p.block_size)) * p.dp;
  const int eb = p.exp_tables[(size_t)seq * p.exp_max_blocks + kp / kExpandBlock], off = kp % kExpandBlock;
  pi_grid_dependency_wait();
  for (int x = tid; x < p.rp / 8; x += 128) reinterpret_cast<uint4*>(p.keys + (size_t)i * p.rp)[x] = reinterpret_cast<const uint4*>(src)[x];
  const int w = p.dpk - p.dim;
  for (int x = tid; x < p.heads * w; x += 128) {
    const int h = x / w, d = x - h * w;
    p.pool[((size_t)eb * p.heads + h) * ((size_t)kExpandBlock * (p.dpk + p.vpk)) + (size_t)off * p.dpk + p.dim + d] =
        d < p.rot ? src[p.rp + d] : __float2bfloat16_rn(0.f);
  }
}

int expanded_dp(const pi_latent_attention& a) { return (a.dim + a.rot_dims + 15) / 16 * 16; }
int expanded_vp(const pi_latent_attention& a) { return (a.vdim + 15) / 16 * 16; }

typedef void (*LatentKernel)(const LatentParams);
cudaError_t grant(pi_ctx* ctx, LatentKernel k, size_t smem) {   // a kernel's shared-memory limit is raised once per device
  static std::vector<std::pair<LatentKernel, pi_smem_grant>> granted;
  if (smem <= kSmemFree) return cudaSuccess;
  for (auto& g : granted)
    if (g.first == k) {
      if (g.second.of(ctx) >= smem) return cudaSuccess;
      g.second.of(ctx) = smem;
      return cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    }
  granted.push_back({k, pi_smem_grant()});
  granted.back().second.of(ctx) = smem;
  return cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

// Clusters of 16 CTAs have to be asked for, once per kernel and device.
pi_status allow_wide_clusters(pi_ctx* ctx, LatentKernel k) {
  static std::vector<std::pair<LatentKernel, int>> done;
  for (auto& d : done)
    if (d.first == k && d.second == ctx->device) return PI_OK;
  PI_CUDA(ctx, cudaFuncSetAttribute(k, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
  done.push_back({k, ctx->device});
  return PI_OK;
}

// Clusters of `splits` CTAs the device holds at once.
int max_clusters(pi_ctx* ctx, LatentKernel k, size_t smem, int splits) {
  struct Known {
    LatentKernel k;
    size_t smem;
    int splits, device, n;
  };
  static std::vector<Known> known;
  for (const Known& c : known)
    if (c.k == k && c.smem == smem && c.splits == splits && c.device == ctx->device) return c.n;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(splits);
  cfg.blockDim = dim3(kDecThreads);
  cfg.dynamicSmemBytes = smem;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = splits;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  int n = 0;
  if (cudaOccupancyMaxActiveClusters(&n, k, &cfg) != cudaSuccess) {
    cudaGetLastError();
    n = 0;
  }
  known.push_back({k, smem, splits, ctx->device, n});
  return n;
}

constexpr int kMaxDecodeDp = 704;
LatentKernel pick_decode(int dp, int rp) {
  if (rp <= 256 && dp <= 192) return latent_decode_kernel<3, 1>;
  if (rp <= 256 && dp <= 384) return latent_decode_kernel<6, 1>;
  if (rp <= 512 && dp <= 576) return latent_decode_kernel<9, 2>;
  return rp <= 512 ? latent_decode_kernel<12, 2> : latent_decode_kernel<12, 4>;
}

}  // namespace

size_t pi_latent_pool_elems(const pi_latent_attention& a, int blocks) {
  return (size_t)blocks * a.heads * kExpandBlock * (expanded_dp(a) + expanded_vp(a));
}
bool pi_latent_expandable(const pi_ctx* ctx, const pi_latent_attention& a, int compute) {
  return compute == PI_BF16 && ctx->opt_tensor_gemm && a.dim % 2 == 0 && expanded_dp(a) <= 256 && expanded_vp(a) <= 256;
}
bool pi_latent_supported(const pi_ctx* ctx, const pi_latent_attention& a, int compute) {
  const int rp = pi_latent_rp(a.rank), dp = pi_latent_dp(a.rank, a.rot_dims);
  if (compute == PI_F32) return ((size_t)dp + 4 * a.rank) * sizeof(float) <= kSmemFit && (size_t)a.dim * sizeof(float) <= kSmemFit;
  return dp <= kMaxDecodeDp && decode_smem(dp, rp).total + 4096 <= ctx->smem_optin && std::max(head_smem(a.dim), head_smem(a.rank)) + 1024 <= ctx->smem_optin;
}

pi_status pi_launch_latent_attention(pi_ctx* ctx, const pi_latent_attention& a, const pi_kv_view& kv, float* proj, size_t stride, void* out,
                                     size_t out_stride, int out_kind, const pi_seq_batch& b, const pi_latent_scratch& s) {
  const bool f32 = kv.kind == PI_F32;
  LatentParams p = {};
  p.proj = proj;
  p.stride = stride;
  p.heads = a.heads;
  p.dim = a.dim;
  p.rot = a.rot_dims;
  p.vdim = a.vdim;
  p.rank = a.rank;
  p.rp = pi_latent_rp(a.rank);
  p.dp = kv.dp;
  p.window = a.window;
  p.block_size = kv.block_size;
  p.block_shift = -1;
  for (int i = 0; i < 31; ++i)
    if (1 << i == kv.block_size) p.block_shift = i;
  p.col_q = a.col_q;
  p.col_kv = a.col_kv;
  p.col_g = a.col_g;
  p.scale = a.scale;
  p.eps = a.eps;
  p.norm = a.norm;
  p.rope_cos = a.rope_cos;
  p.rope_sin = a.rope_sin;
  p.uk_t = a.uk_t->w;
  p.uk_ld = a.uk_t->ld;
  p.uv_ld = a.ukv->ld;
  p.uv = static_cast<const uint16_t*>(a.ukv->w) + (size_t)a.heads * a.dim * a.ukv->ld;
  p.q = s.q;
  p.o = s.o;
  p.base = kv.base;
  p.out = out;
  p.out_stride = out_stride;
  p.row_seq = b.row_seq;
  p.row_pos = b.row_pos;
  p.seq_n = b.seq_n;
  p.seq_start = b.seq_start;
  p.lens = b.lens;
  p.tables = b.tables;
  p.max_blocks = b.max_blocks;
  p.rows = b.rows;
  p.latent_rows = b.latent_rows;
  p.n_latent = b.n_latent;
  p.expand_min = b.n_expand ? kExpandPortion : INT_MAX;
  p.slices = (a.rank + kHeadCols - 1) / kHeadCols;
  const int row_tiles = (b.n_latent + kHeadRows - 1) / kHeadRows;
  p.row_splits = std::max(1, std::min(row_tiles, 2 * ctx->sm_count / std::max(1, a.heads * p.slices)));
  {
    pi_prof_scope prof(ctx, PI_PROF_ROPE_KV);
    const LatentKernel k = f32 ? latent_prepare_kernel<float> : latent_prepare_kernel<__nv_bfloat16>;
    const size_t smem = f32 ? (size_t)a.dim * sizeof(float) : head_smem(a.dim);
    PI_CUDA(ctx, grant(ctx, k, smem));
    const int absorb = b.n_latent == 0 ? 0 : f32 ? b.n_latent * a.heads : a.heads * p.slices * p.row_splits;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(b.rows + absorb), dim3(kHeadThreads), smem, 1, p));
  }
  if (b.n_latent > 0 && f32) {
    pi_maps_attention m;
    m.heads = a.heads;
    m.kv_heads = 1;
    m.dim = kv.dp;
    m.vdim = a.rank;
    m.window = a.window;
    m.scale = a.scale;
    m.v_in_k = true;
    PI_TRY(pi_launch_maps_attention(ctx, m, kv, static_cast<const float*>(s.q), (size_t)a.heads * kv.dp, s.o, (size_t)a.heads * a.rank, PI_F32, b));
    pi_prof_scope prof(ctx, PI_PROF_ATTENTION);
    const LatentKernel k = out_kind == PI_BF16 ? latent_out_f32_kernel<__nv_bfloat16> : latent_out_f32_kernel<float>;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(a.heads, b.n_latent), dim3(kHeadThreads), (size_t)a.rank * sizeof(float), 1, p));
  } else if (b.n_latent > 0) {
    p.groups = (a.heads + 15) / 16;
    const LatentKernel k = pick_decode(p.dp, p.rp);
    const size_t smem = decode_smem(p.dp, p.rp).total;
    PI_CUDA(ctx, grant(ctx, k, smem));
    PI_TRY(allow_wide_clusters(ctx, k));
    // KV splits: one round of CTAs over the GPU, at least a tile each
    const int keys = a.window > 0 ? std::min(a.window, b.max_pos + 1) : b.max_pos + 1;
    const long ctas = (long)b.n_latent * p.groups, tiles = (keys + kKeys - 1) / kKeys;
    p.nsplit = (int)std::max(1L, std::min({(long)ctx->sm_count / ctas, tiles, (long)kMaxSplits}));
    while (p.nsplit > 1 && ctas > max_clusters(ctx, k, smem, p.nsplit)) --p.nsplit;
    {
      pi_prof_scope prof(ctx, PI_PROF_ATTENTION);
      PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(p.nsplit, b.n_latent, p.groups), dim3(kDecThreads), smem, p.nsplit, p));
    }
    pi_prof_scope prof(ctx, PI_PROF_ROPE_KV);
    const LatentKernel ko = out_kind == PI_BF16 ? latent_out_kernel<__nv_bfloat16> : latent_out_kernel<float>;
    const size_t so = head_smem(a.rank);
    PI_CUDA(ctx, grant(ctx, ko, so));
    const int slices = (a.vdim + kHeadCols - 1) / kHeadCols;
    const int z = std::max(1, std::min(row_tiles, 2 * ctx->sm_count / (a.heads * slices)));
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, ko, dim3(slices, a.heads, z), dim3(kHeadThreads), so, 1, p));
  }
  if (b.n_expand > 0) {
    const int dpk = expanded_dp(a), vpk = expanded_vp(a);
    const GatherParams g = {static_cast<const __nv_bfloat16*>(kv.base), kv.dp, p.rp, a.rank, a.rot_dims, kv.block_size, b.key_seq, b.key_pos, b.exp_lo, b.tables,
                            b.max_blocks, b.exp_tables, b.exp_max_blocks, s.keys, s.pool, a.heads, a.dim, dpk, vpk};
    {
      pi_prof_scope prof(ctx, PI_PROF_ROPE_KV);
      PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, latent_gather_kernel, dim3(b.n_keys), dim3(128), 0, 1, g));
    }
    pi_maps_kv mk;
    mk.k_rows = a.heads * a.dim;
    mk.dim = a.dim;
    mk.vdim = a.vdim;
    mk.base = s.pool;
    mk.kind = PI_BF16;
    mk.kv_heads = a.heads;
    mk.dp = dpk;
    mk.vp = vpk;
    mk.block_size = kExpandBlock;
    mk.row_seq = b.key_seq;
    mk.row_pos = b.key_pos;
    mk.lens = b.exp_lens;
    mk.tables = b.exp_tables;
    mk.max_blocks = b.exp_max_blocks;
    pi_linear_args g2;
    g2.M = b.n_keys;
    g2.x_bf16 = s.keys;
    g2.x_stride = p.rp;
    g2.epi = PI_EPI_MAPS_QKV;
    g2.maps_kv = &mk;
    PI_TRY(pi_launch_gemm_bf16(ctx, a.ukv, g2));
    pi_maps_attention m;
    m.heads = m.kv_heads = a.heads;
    m.dim = a.dim + a.rot_dims;
    m.vdim = a.vdim;
    m.window = a.window;
    m.scale = a.scale;
    m.gate = proj + a.col_g;
    m.gate_stride = stride;
    pi_kv_view v;
    v.base = s.pool;
    v.kind = PI_BF16;
    v.kv_heads = a.heads;
    v.maps = 1;
    v.dp = dpk;
    v.vp = vpk;
    v.block_size = kExpandBlock;
    pi_seq_batch e = b;
    e.n_single = 0;
    e.portions = b.expand;
    e.n_portions = b.n_expand;
    e.max_portion = b.max_expand;
    e.seq_start = b.exp_start;
    e.lens = b.exp_lens;
    e.tables = b.exp_tables;
    e.max_blocks = b.exp_max_blocks;
    PI_TRY(pi_launch_maps_attention(ctx, m, v, proj + a.col_q, stride, out, out_stride, out_kind, e));
  }
  return PI_OK;
}
