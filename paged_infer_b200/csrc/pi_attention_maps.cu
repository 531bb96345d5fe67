// Windowed attention with one or two softmax maps per head over the same values (differential attention), reading the
// paged KV pool.
//
//   score_j = scale (q_j . k_j) - slope (t - s)     j = map, over the keys t - window < s <= t; slope: of the head, if there is one
//   a_j     = softmax(score_j) V          (with a sink, exp(sink) is one more term of the denominator)
//   out     = a_1                                             (one map)
//   o = a_1 - lambda a_2;  out = out_scale o / rms(o)          (two maps)
//   out *= sigmoid(gate)                                       (with an output gate, per channel or per head)
//
// or, with one map, keys that weigh by themselves: a_1 = sum over the keys of sigmoid(score_1 + bias of the head) v.
//
// Kernels: maps_prepare_kernel brings q, k and v into their final form (bias, unit root mean square, rotation, temperature of the
// queries, mixing of the values) and writes k and v into the pool; maps_prepare_whole_kernel is the one for q and k that are
// normalised over the whole projection; maps_attn_plain_kernel is the f32
// path and the one for sizes the tensor-core kernels of pi_attention_maps_tc.cu do not hold.
#include <math.h>

#include <algorithm>

#include "pi_attention_maps.cuh"

namespace {

struct PrepareParams {
  float* qkv;
  size_t stride;
  int heads, kv_heads, maps, dim, vdim, rot_dims;
  const float *rope_cos, *rope_sin;
  void* base;
  int dp, vp, block_size;
  const int32_t *row_seq, *row_pos, *lens, *tables;
  int max_blocks;
  float eps;
  pi_maps_prepare x;
};

template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v);
template <>
__device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <>
__device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

// Warp per vector of a row: a q or k vector of one map, or a head's values.  Lanes hold groups of adjacent channels (rot_dims is
// even, so a rotation pair stays together): four (VEC: sizes are multiples of 4, at most 256), or two, up to kHeld of them in
// registers, longer vectors are read twice.  Pool rows are padded with zeros up to dp / vp.
constexpr int kPrepareWarps = 4, kHeld = 4;
template <typename T, bool VEC>
__global__ void __launch_bounds__(kPrepareWarps * 32) maps_prepare_kernel(const PrepareParams p) {
  const int row = blockIdx.x, lane = threadIdx.x & 31, vec = blockIdx.y * kPrepareWarps + (threadIdx.x >> 5);
  const int nq = p.heads * p.maps, nk = p.kv_heads * p.maps, half = p.rot_dims >> 1;
  const bool is_q = vec < nq;
  const int pos = p.row_pos[row], off = pos % p.block_size;
  bool mapped = false;
  int pb = 0;
  if (!is_q) {
    const int seq = p.row_seq[row], lb = pos / p.block_size;
    mapped = lb < p.lens[seq];
    if (mapped) pb = p.tables[(size_t)seq * p.max_blocks + lb];
  }
  pi_grid_dependency_wait();
  if (vec >= nq + nk + p.kv_heads) return;
  const size_t tile = (size_t)p.block_size * (p.maps * p.dp + p.vp);
  if (vec >= nq + nk) {
    const int g = vec - nq - nk, at = (nq + nk) * p.dim + g * p.vdim;
    const float* v = p.qkv + (size_t)row * p.stride + at;
    T* dst = static_cast<T*>(p.base) + ((size_t)pb * p.kv_heads + g) * tile + (size_t)p.block_size * p.maps * p.dp + (size_t)off * p.vp;
    if (VEC) {
      for (int e = lane * 4; e < p.vp; e += 128) {
        float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
        if (e < p.vdim) {
          r = *reinterpret_cast<const float4*>(v + e);
          if (p.x.bias) {
            const float4 b = __ldg(reinterpret_cast<const float4*>(p.x.bias + at + e));
            r = make_float4(r.x + b.x, r.y + b.y, r.z + b.z, r.w + b.w);
          }
          const pi_value_mix& m = p.x.mix;
          if (m.first) {
            float4* f = reinterpret_cast<float4*>(m.first + (size_t)row * m.stride + g * p.vdim + e);
            if (m.keeps) {
              *f = r;
            } else {
              const float4 o = *f;
              const float l = m.lambda, k = 1.f - l;
              r = make_float4(fmaf(l, o.x, k * r.x), fmaf(l, o.y, k * r.y), fmaf(l, o.z, k * r.z), fmaf(l, o.w, k * r.w));
            }
          }
        }
        if (mapped) store4<T>(dst + e, r);
      }
      return;
    }
    for (int e = lane; e < p.vp; e += 32) {
      float r = 0.f;
      if (e < p.vdim) r = pi_mix_value(p.x.mix, row, g * p.vdim + e, v[e] + (p.x.bias ? __ldg(p.x.bias + at + e) : 0.f));
      if (mapped) dst[e] = pi_from_f32<T>(r);
    }
    return;
  }
  const int pairs = (p.dp + 1) >> 1;     // dp >= dim, the pad is written too
  float* v = p.qkv + (size_t)row * p.stride + (size_t)vec * p.dim;   // k vectors follow the q vectors
  const float* bias = p.x.bias ? p.x.bias + (size_t)vec * p.dim : nullptr;
  const int kv = vec - nq, kg = is_q ? 0 : kv / p.maps, km = kv - kg * p.maps;
  T* dst = static_cast<T*>(p.base) + ((size_t)pb * p.kv_heads + kg) * tile + (size_t)off * p.maps * p.dp + (size_t)km * p.dp;
  const float* cs = p.rope_cos + (size_t)pos * half;
  const float* sn = p.rope_sin + (size_t)pos * half;
  float factor = is_q && p.x.q_temp ? __ldg(p.x.q_temp + pos) : 1.f;
  if (VEC) {
    float4 c[2];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int d = lane * 4 + 128 * i;
      c[i] = d < p.dim ? *reinterpret_cast<const float4*>(v + d) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (bias && d < p.dim) {
        const float4 b = __ldg(reinterpret_cast<const float4*>(bias + d));
        c[i] = make_float4(c[i].x + b.x, c[i].y + b.y, c[i].z + b.z, c[i].w + b.w);
      }
      ss = fmaf(c[i].x, c[i].x, fmaf(c[i].y, c[i].y, fmaf(c[i].z, c[i].z, fmaf(c[i].w, c[i].w, ss))));
    }
    if (p.x.unit_qk) factor /= sqrtf(pi_warp_sum(ss) / (float)p.dim + p.eps);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int d = lane * 4 + 128 * i, j = d >> 1;
      float4 r = c[i];
      if (j < half) {
        r.x = c[i].x * cs[j] - c[i].y * sn[j];
        r.y = c[i].y * cs[j] + c[i].x * sn[j];
      }
      if (j + 1 < half) {
        r.z = c[i].z * cs[j + 1] - c[i].w * sn[j + 1];
        r.w = c[i].w * cs[j + 1] + c[i].z * sn[j + 1];
      }
      r = make_float4(r.x * factor, r.y * factor, r.z * factor, r.w * factor);
      if (is_q) {
        if (d < p.dim) *reinterpret_cast<float4*>(v + d) = r;
      } else if (mapped && d < p.dp) {
        store4<T>(dst + d, r);
      }
    }
    return;
  }
  auto load = [&](int j) {
    const int d = 2 * j;
    float2 c = make_float2(d < p.dim ? v[d] : 0.f, d + 1 < p.dim ? v[d + 1] : 0.f);
    if (bias) {
      if (d < p.dim) c.x += __ldg(bias + d);
      if (d + 1 < p.dim) c.y += __ldg(bias + d + 1);
    }
    return c;
  };
  float2 held[kHeld];
#pragma unroll
  for (int i = 0; i < kHeld; ++i) held[i] = lane + 32 * i < pairs ? load(lane + 32 * i) : make_float2(0.f, 0.f);
  if (p.x.unit_qk) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kHeld; ++i) ss = fmaf(held[i].x, held[i].x, fmaf(held[i].y, held[i].y, ss));
    for (int j = lane + 32 * kHeld; j < pairs; j += 32) {
      const float2 c = load(j);
      ss = fmaf(c.x, c.x, fmaf(c.y, c.y, ss));
    }
    factor /= sqrtf(pi_warp_sum(ss) / (float)p.dim + p.eps);
  }
  auto finish = [&](int j, float2 c) {
    const int d = 2 * j;
    if (j < half) c = make_float2(c.x * cs[j] - c.y * sn[j], c.y * cs[j] + c.x * sn[j]);
    c.x *= factor;
    c.y *= factor;
    if (is_q) {
      if (d < p.dim) v[d] = c.x;
      if (d + 1 < p.dim) v[d + 1] = c.y;
    } else if (mapped) {
      dst[d] = pi_from_f32<T>(c.x);
      dst[d + 1] = pi_from_f32<T>(c.y);
    }
  };
#pragma unroll
  for (int i = 0; i < kHeld; ++i)
    if (lane + 32 * i < pairs) finish(lane + 32 * i, held[i]);
  for (int j = lane + 32 * kHeld; j < pairs; j += 32) finish(j, load(j));
}

// CTA per row: q and k (which follow one another) each over the root mean square of all their heads, times a weight per channel, then
// rotated; v as it is.  Groups of four adjacent channels (VEC: sizes are multiples of 4) or pairs, up to kWholeHeld of them per thread
// in registers, the others are read twice.  Pool rows are padded with zeros up to dp / vp.
constexpr int kWholeHeld = 5;
template <typename T, bool VEC, int THREADS>
__global__ void __launch_bounds__(THREADS) maps_prepare_whole_kernel(const PrepareParams p) {
  constexpr int G = VEC ? 4 : 2;
  __shared__ float red[2][THREADS / 32];
  const int row = blockIdx.x, tid = threadIdx.x, half = p.rot_dims >> 1;
  const int gd = (p.dim + G - 1) / G, nq = p.heads * gd, n = nq + (p.x.q_only ? 0 : p.kv_heads * gd);   // groups: of a head, of q, of all
  const int pos = p.row_pos[row], off = pos % p.block_size;
  bool mapped = false;
  int pb = 0;
  if (!p.x.q_only) {
    const int seq = p.row_seq[row], lb = pos / p.block_size;
    mapped = lb < p.lens[seq];
    if (mapped) pb = p.tables[(size_t)seq * p.max_blocks + lb];
  }
  const float* cs = p.rope_cos + (size_t)pos * half;
  const float* sn = p.rope_sin + (size_t)pos * half;
  float* qkv = p.qkv + (size_t)row * p.stride;
  struct Group {
    float v[G];
  };
  auto load = [&](const float* src, int i) {
    Group g;
    if (VEC) {                            // no group is ragged
      const float4 f = reinterpret_cast<const float4*>(src)[i];
      g.v[0] = f.x;
      g.v[1] = f.y;
      g.v[G - 2] = f.z;
      g.v[G - 1] = f.w;
    } else {
      const int vec = i / gd, d = (i - vec * gd) * G;
      src += (size_t)vec * p.dim + d;
      g.v[0] = src[0];
      g.v[1] = d + 1 < p.dim ? src[1] : 0.f;
    }
    return g;
  };
  auto square = [&](const Group& g) {
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < G; ++k) s = fmaf(g.v[k], g.v[k], s);
    return s;
  };
  Group w[kWholeHeld];                    // constants: ahead of the dependency wait
#pragma unroll
  for (int j = 0; j < kWholeHeld; ++j) w[j] = load(p.x.norm_qk, min(tid + j * THREADS, n - 1));
  pi_grid_dependency_wait();
  Group held[kWholeHeld];
  float ss[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < kWholeHeld; ++j) held[j] = load(qkv, min(tid + j * THREADS, n - 1));
#pragma unroll
  for (int j = 0; j < kWholeHeld; ++j) {
    const int i = tid + j * THREADS;
    if (i < nq) ss[0] += square(held[j]);
    else if (i < n) ss[1] += square(held[j]);
  }
  for (int i = tid + kWholeHeld * THREADS; i < n; i += THREADS) ss[i < nq ? 0 : 1] += square(load(qkv, i));
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    ss[k] = pi_warp_sum(ss[k]);
    if ((tid & 31) == 0) red[k][tid >> 5] = ss[k];
  }
  // the values do not wait for the sums
  const size_t tile = (size_t)p.block_size * (p.dp + p.vp);
  T* blk = static_cast<T*>(p.base) + (size_t)pb * p.kv_heads * tile;
  if (mapped) {
    const float* v = qkv + (size_t)(p.heads + p.kv_heads) * p.dim;
    for (int i = tid; i < p.kv_heads * (p.vp / G); i += THREADS) {
      const int g = i / (p.vp / G), e = (i - g * (p.vp / G)) * G;
      T* dst = blk + g * tile + (size_t)p.block_size * p.dp + (size_t)off * p.vp + e;
      if (VEC) {
        store4<T>(dst, e < p.vdim ? *reinterpret_cast<const float4*>(v + (size_t)g * p.vdim + e) : make_float4(0.f, 0.f, 0.f, 0.f));
      } else {
#pragma unroll
        for (int k = 0; k < G; ++k) dst[k] = pi_from_f32<T>(e + k < p.vdim ? v[(size_t)g * p.vdim + e + k] : 0.f);
      }
    }
    for (int i = tid; i < p.kv_heads * (p.dp - p.dim); i += THREADS) {
      const int g = i / (p.dp - p.dim), d = p.dim + i - g * (p.dp - p.dim);
      blk[g * tile + (size_t)off * p.dp + d] = pi_from_f32<T>(0.f);
    }
  }
  __syncthreads();
  float inv[2] = {0.f, 0.f};
#pragma unroll
  for (int k = 0; k < 2; ++k) {
#pragma unroll
    for (int j = 0; j < THREADS / 32; ++j) inv[k] += red[k][j];
    inv[k] = 1.0f / sqrtf(inv[k] / (float)((k ? p.kv_heads : p.heads) * p.dim) + p.eps);
  }
  auto finish = [&](int i, Group g, const Group& w) {
    const int vec = i / gd, d = (i - vec * gd) * G;
    const float f = inv[i < nq ? 0 : 1];
#pragma unroll
    for (int k = 0; k < G; ++k) g.v[k] = g.v[k] * f * w.v[k];
#pragma unroll
    for (int k = 0; k < G; k += 2) {
      const int j = (d + k) >> 1;
      if (j < half) {
        const float a = g.v[k], b = g.v[k + 1];
        g.v[k] = a * cs[j] - b * sn[j];
        g.v[k + 1] = b * cs[j] + a * sn[j];
      }
    }
    if (i < nq) {
      float* dst = qkv + (size_t)vec * p.dim + d;
      if (VEC) {
        *reinterpret_cast<float4*>(dst) = make_float4(g.v[0], g.v[1], g.v[G - 2], g.v[G - 1]);
      } else {
        dst[0] = g.v[0];
        if (d + 1 < p.dim) dst[1] = g.v[1];
      }
    } else if (mapped) {
      T* dst = blk + (vec - p.heads) * tile + (size_t)off * p.dp + d;
      if (VEC) {
        store4<T>(dst, make_float4(g.v[0], g.v[1], g.v[G - 2], g.v[G - 1]));
      } else {
        dst[0] = pi_from_f32<T>(g.v[0]);
        if (d + 1 < p.dim) dst[1] = pi_from_f32<T>(g.v[1]);
      }
    }
  };
#pragma unroll
  for (int j = 0; j < kWholeHeld; ++j)
    if (tid + j * THREADS < n) finish(tid + j * THREADS, held[j], w[j]);
  for (int i = tid + kWholeHeld * THREADS; i < n; i += THREADS) finish(i, load(qkv, i), load(p.x.norm_qk, i));
}

// One CTA of 4 warps per (row, head): the warps take every fourth key and merge; lanes hold the channels.  f32
// throughout, any sizes (smem: q, per-warp accumulators of both maps).
constexpr int kPlainWarps = 4;
template <typename T, typename O>
__global__ void __launch_bounds__(kPlainWarps * 32) maps_attn_plain_kernel(const MapsParams p) {
  extern __shared__ float sm[];
  const int row = blockIdx.y, head = blockIdx.x, g = head / (p.heads / p.kv_heads);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = p.row_seq[row], pos = p.row_pos[row], len = p.lens[seq];
  const int32_t* table = p.tables + (size_t)seq * p.max_blocks;
  const int nm = p.maps, DP = p.dp;
  float* sq = sm;                                   // [maps][dim]
  float* acc = sm + nm * p.dim;                     // [warps][maps][vdim]
  __shared__ float s_m[kPlainWarps][2], s_l[kPlainWarps][2], s_red[kPlainWarps];
  pi_grid_dependency_wait();
  for (int i = tid; i < nm * p.dim; i += blockDim.x) sq[i] = p.q[(size_t)row * p.stride + (size_t)head * nm * p.dim + i];
  float* my = acc + (size_t)warp * nm * p.vdim;
  for (int i = lane; i < nm * p.vdim; i += 32) my[i] = 0.f;
  __syncthreads();
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const size_t tile = (size_t)p.block_size * (nm * DP + p.vp);
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float slope = p.slopes ? __ldg(p.slopes + head) : 0.f, sink = p.sinks ? __ldg(p.sinks + head) : -INFINITY;
  const bool by_itself = p.sigmoid_bias != nullptr;
  const float self_bias = by_itself ? __ldg(p.sigmoid_bias + head) : 0.f;
  for (int t = lo + warp; t <= pos; t += kPlainWarps) {
    const int lb = t / p.block_size, off = t - lb * p.block_size;
    if (lb >= len) break;
    const T* kt = static_cast<const T*>(p.base) + ((size_t)table[lb] * p.kv_heads + g) * tile;
    const T* vt = kt + (size_t)p.block_size * nm * DP + (size_t)off * p.vp;
    kt += (size_t)off * nm * DP;
    if (p.v_in_k) vt = kt;
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      if (m >= nm) break;
      float d = 0.f;
      for (int i = lane; i < p.dim; i += 32) d = fmaf(sq[m * p.dim + i], pi_to_f32(kt[m * DP + i]), d);
      const float s = pi_warp_sum(d) * p.scale - slope * (float)(pos - t);
      if (by_itself) {
        const float w = pi_sigmoid(s + self_bias);
        for (int i = lane; i < p.vdim; i += 32) my[i] = fmaf(w, pi_to_f32(vt[i]), my[i]);
        continue;
      }
      const float mn = fmaxf(mx[m], s), keep = expf(mx[m] - mn), w = expf(s - mn);
      mx[m] = mn;
      l[m] = l[m] * keep + w;
      for (int i = lane; i < p.vdim; i += 32) my[m * p.vdim + i] = my[m * p.vdim + i] * keep + w * pi_to_f32(vt[i]);
    }
  }
  if (lane == 0)
    for (int m = 0; m < nm; ++m) {
      s_m[warp][m] = mx[m];
      s_l[warp][m] = l[m];
    }
  __syncthreads();
  float f[2][kPlainWarps];
  for (int m = 0; m < nm; ++m) {
    float M = sink, L = 0.f;
    for (int w = 0; w < kPlainWarps; ++w) M = fmaxf(M, s_m[w][m]);
    if (p.sinks) L = expf(sink - M);
    for (int w = 0; w < kPlainWarps; ++w) L += s_m[w][m] == -INFINITY ? 0.f : s_l[w][m] * expf(s_m[w][m] - M);
    for (int w = 0; w < kPlainWarps; ++w) f[m][w] = by_itself ? 1.f : s_m[w][m] == -INFINITY ? 0.f : expf(s_m[w][m] - M) / L;
  }
  float sq_sum = 0.f;
  for (int e = tid; e < p.vdim; e += blockDim.x) {
    float a[2] = {0.f, 0.f};
    for (int m = 0; m < nm; ++m)
      for (int w = 0; w < kPlainWarps; ++w) a[m] += acc[((size_t)w * nm + m) * p.vdim + e] * f[m][w];
    const float o = nm == 2 ? a[0] - p.lambda * a[1] : a[0];
    sq_sum = fmaf(o, o, sq_sum);
    acc[e] = o;   // warp 0, map 0: this thread is the only one that reads column e
  }
  float r = 1.0f;
  if (nm == 2) {
    sq_sum = pi_warp_sum(sq_sum);
    if (lane == 0) s_red[warp] = sq_sum;
    __syncthreads();
    float t = 0.f;
    for (int w = 0; w < kPlainWarps; ++w) t += s_red[w];
    r = p.out_scale / sqrtf(t / (float)p.vdim + p.eps);
  }
  O* o = static_cast<O*>(p.out) + (size_t)row * p.out_stride + (size_t)head * p.vdim;
  const float* gate = p.gate ? p.gate + (size_t)row * p.gate_stride + (p.gate_per_head ? head : (size_t)head * p.vdim) : nullptr;
  for (int e = tid; e < p.vdim; e += blockDim.x) o[e] = pi_from_f32<O>(acc[e] * (gate ? r * pi_sigmoid(gate[p.gate_per_head ? 0 : e]) : r));
}

}  // namespace

pi_status pi_launch_maps_prepare(pi_ctx* ctx, const pi_maps_attention& a, const pi_maps_prepare& x, const pi_kv_view& kv, float* qkv, size_t stride,
                                 const pi_seq_batch& b) {
  pi_prof_scope prof(ctx, PI_PROF_ROPE_KV);
  PrepareParams p = {qkv, stride, a.heads, a.kv_heads, a.maps, a.dim, a.vdim, a.rot_dims, a.rope_cos, a.rope_sin, kv.base, kv.dp, kv.vp,
                     kv.block_size, b.row_seq, b.row_pos, b.lens, b.tables, b.max_blocks, a.eps, x};
  const int vectors = (a.heads + a.kv_heads) * a.maps + a.kv_heads;
  const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.dim <= 256 && a.vdim <= 256 && stride % 4 == 0 && x.mix.stride % 4 == 0;
  if (x.norm_qk) {
    PI_REQUIRE(ctx, a.maps == 1 && !x.bias && !x.unit_qk && !x.q_temp && !x.mix.first, "norms over whole projections stand alone");
    const int groups = (a.heads + (x.q_only ? 0 : a.kv_heads)) * ((a.dim + (vec ? 3 : 1)) / (vec ? 4 : 2)), threads = groups <= 128 * kWholeHeld && b.rows > ctx->sm_count ? 128 : 256;
    auto pick = [&](auto few, auto many) { return threads == 128 ? few : many; };
    void (*k)(const PrepareParams);
    if (kv.kind == PI_BF16) k = vec ? pick(maps_prepare_whole_kernel<__nv_bfloat16, true, 128>, maps_prepare_whole_kernel<__nv_bfloat16, true, 256>)
                                    : pick(maps_prepare_whole_kernel<__nv_bfloat16, false, 128>, maps_prepare_whole_kernel<__nv_bfloat16, false, 256>);
    else k = vec ? pick(maps_prepare_whole_kernel<float, true, 128>, maps_prepare_whole_kernel<float, true, 256>)
                 : pick(maps_prepare_whole_kernel<float, false, 128>, maps_prepare_whole_kernel<float, false, 256>);
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(b.rows), dim3(threads), 0, 1, p));
    return PI_OK;
  }
  PI_REQUIRE(ctx, !x.q_only, "keys of another layer go with norms over whole projections");
  void (*k)(const PrepareParams);
  if (kv.kind == PI_BF16) k = vec ? maps_prepare_kernel<__nv_bfloat16, true> : maps_prepare_kernel<__nv_bfloat16, false>;
  else k = vec ? maps_prepare_kernel<float, true> : maps_prepare_kernel<float, false>;
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(b.rows, (vectors + kPrepareWarps - 1) / kPrepareWarps), dim3(kPrepareWarps * 32), 0, 1, p));
  return PI_OK;
}

pi_status pi_launch_maps_attention(pi_ctx* ctx, const pi_maps_attention& a, const pi_kv_view& kv, const float* qkv, size_t stride,
                                   void* out, size_t out_stride, int out_kind, const pi_seq_batch& b) {
  pi_prof_scope prof(ctx, PI_PROF_ATTENTION);
  MapsParams p = {qkv, stride, out, out_stride, kv.base, a.heads, a.kv_heads, a.maps, a.dim, a.vdim, kv.dp, kv.vp, kv.block_size,
                  a.window, a.scale, a.eps, a.lambda, a.out_scale, b.row_seq, b.row_pos, b.lens, b.tables, b.max_blocks, a.gate, a.gate_stride, a.gate_per_head,
                  a.slopes, a.sinks, a.sigmoid_bias, a.v_in_k};
  PI_REQUIRE(ctx, !a.sigmoid_bias || (a.maps == 1 && !a.slopes && !a.sinks), "keys that weigh by themselves go with one map and plain scores");
  if (pi_maps_attention_tc_usable(ctx, a, kv)) return pi_launch_maps_attention_tc(ctx, p, out_kind, b);
  const size_t smem = sizeof(float) * ((size_t)a.maps * a.dim + (size_t)kPlainWarps * a.maps * a.vdim);
  PI_REQUIRE(ctx, smem <= kSmemFit, "attention heads of %d / %d channels are too wide", a.dim, a.vdim);
  auto k = kv.kind == PI_BF16 ? (out_kind == PI_BF16 ? maps_attn_plain_kernel<__nv_bfloat16, __nv_bfloat16> : maps_attn_plain_kernel<__nv_bfloat16, float>)
                              : (out_kind == PI_BF16 ? maps_attn_plain_kernel<float, __nv_bfloat16> : maps_attn_plain_kernel<float, float>);
  // grid.y is limited to 65535 rows, far above any step
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(a.heads, b.rows), dim3(kPlainWarps * 32), smem, 1, p));
  return PI_OK;
}
