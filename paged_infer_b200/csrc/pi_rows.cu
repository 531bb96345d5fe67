// Row-wise steps between sublayers: one CTA per row takes up what the last sublayer left - the embedding, the residual row as
// it is, the sublayer's result, or the outputs of the row's experts - and writes the next sublayer's input.  All sums are f32.
//
// row_norm_kernel: sublayers that are normalised before (layer norm: zero mean, unit variance, a weight, no bias); mean and
// variance are two passes over the row in shared memory.
// row_rms_kernel: sublayers that are normalised before and after: x += rms norm of the result, then h = rms norm of x (or x as it
// stands); or sublayers whose sum is normalised: x = rms norm of (keep x + result).  The result may be gated channel by channel
// first.  The row stays in registers between the two norms.  The embedding may have a row of a table of token pairs beside it.
#include <algorithm>

#include "pi_layered.cuh"

namespace {

constexpr int kRowThreads = 256;

enum RowSource { kFromX, kFromEmbedding, kFromExperts, kFromResult };

struct RowParams {
  float* x;
  int width;
  const int32_t* pick;
  const uint16_t* table;
  size_t table_ld;
  int vocab;
  const uint32_t* tokens;
  pi_expert_sum e;
  const float* w;
  float eps;
  void* h;
  size_t ld_h;
  // RMS norms
  const float* y;
  size_t y_stride;
  const float* post_w;
  float post_eps, embed_scale;
  int of_sum;
  float keep;
  const float *gate, *gate_bias;
  size_t gate_stride;
  pi_token_pairs pairs;
};

__device__ __forceinline__ float row_sum(float v, float* red) {   // over the CTA; the same bits in every thread
  v = pi_warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kRowThreads / 32; ++i) t += red[i];
  return t;
}

__device__ __forceinline__ float expert_value(const pi_expert_sum& e, size_t i) {
  return e.y_bf16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(e.y)[i]) : static_cast<const float*>(e.y)[i];
}
__device__ __forceinline__ float4 expert_value4(const pi_expert_sum& e, size_t i) {
  if (!e.y_bf16) return *reinterpret_cast<const float4*>(static_cast<const float*>(e.y) + i);
  const uint2 u = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(e.y) + i);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ float4 fma4(float a, float4 b, float4 c) {
  return make_float4(fmaf(a, b.x, c.x), fmaf(a, b.y, c.y), fmaf(a, b.z, c.z), fmaf(a, b.w, c.w));
}

template <typename T, RowSource SRC>
__global__ void __launch_bounds__(kRowThreads) row_norm_kernel(const RowParams p) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[kRowThreads / 32];
  __shared__ float s_w[64];
  __shared__ int s_at[64];
  const int r = blockIdx.x, tid = threadIdx.x;
  const int src = p.pick ? p.pick[r] : r;
  if (SRC == kFromEmbedding) pi_grid_dependency_wait_strict();   // the step's fence, see pi_seq_batch
  else pi_grid_dependency_wait();
  float* x = p.x + (size_t)src * p.width;
  float sum = 0.f;
  if (SRC == kFromEmbedding) {
    const uint16_t* t = p.table + (size_t)(p.tokens[r] % (uint32_t)p.vocab) * p.table_ld;
    for (int i = tid; i < p.width; i += kRowThreads) {
      const float v = pi_bf16_bits_to_f32(t[i]);
      x[i] = v;
      row[i] = v;
      sum += v;
    }
  } else if (SRC == kFromExperts) {
    const pi_expert_sum& e = p.e;
    if (tid < e.top) {
      s_w[tid] = e.weights[(size_t)r * e.top + tid];
      s_at[tid] = e.place ? e.place[(size_t)r * e.top + tid] : r * e.top + tid;
    }
    const float gate = e.shared ? pi_sigmoid(e.shared_gate[(size_t)r * e.shared_gate_stride]) : 0.f;
    __syncthreads();
    const int wide = p.width % 4 == 0 ? p.width : 0;   // four channels at a time, four experts' loads in flight
    for (int i = tid * 4; i < wide; i += kRowThreads * 4) {
      const float4 old = *reinterpret_cast<const float4*>(x + i), sc = __ldg(reinterpret_cast<const float4*>(e.scale + i));
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (e.shared) v = fma4(gate, *reinterpret_cast<const float4*>(e.shared + (size_t)r * e.shared_stride + i), v);
      for (int k0 = 0; k0 < e.top; k0 += 4) {
        float4 y[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) y[k] = expert_value4(e, (size_t)s_at[min(k0 + k, e.top - 1)] * e.y_stride + i);
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (k0 + k < e.top) v = fma4(s_w[k0 + k], y[k], v);
      }
      v = make_float4(fmaf(sc.x, v.x, old.x), fmaf(sc.y, v.y, old.y), fmaf(sc.z, v.z, old.z), fmaf(sc.w, v.w, old.w));
      *reinterpret_cast<float4*>(x + i) = v;
      *reinterpret_cast<float4*>(row + i) = v;
      sum += (v.x + v.y) + (v.z + v.w);
    }
    for (int i = wide + tid; i < p.width; i += kRowThreads) {
      float v = e.shared ? gate * e.shared[(size_t)r * e.shared_stride + i] : 0.f;
      for (int k = 0; k < e.top; ++k) v = fmaf(s_w[k], expert_value(e, (size_t)s_at[k] * e.y_stride + i), v);
      v = fmaf(e.scale[i], v, x[i]);
      x[i] = v;
      row[i] = v;
      sum += v;
    }
  } else {
    for (int i = tid; i < p.width; i += kRowThreads) {
      const float v = x[i];
      row[i] = v;
      sum += v;
    }
  }
  if (!p.h) return;
  if (SRC == kFromExperts) __syncthreads();
  const float mean = row_sum(sum, red) / (float)p.width;
  float sq = 0.f;
  for (int i = tid; i < p.width; i += kRowThreads) {
    const float d = row[i] - mean;
    sq = fmaf(d, d, sq);
  }
  const float inv = 1.0f / sqrtf(row_sum(sq, red) / (float)p.width + p.eps);
  T* h = static_cast<T*>(p.h) + (size_t)r * p.ld_h;
  for (int i = tid; i < p.width; i += kRowThreads) h[i] = pi_from_f32<T>((row[i] - mean) * inv * __ldg(p.w + i));
}

// Sum over the CTA's 256 threads with one barrier; `red` must not have been used since the barrier before last.
__device__ __forceinline__ float row_sum_once(float v, float* red) {
  v = pi_warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kRowThreads / 32; ++i) t += red[i];
  return t;
}
__device__ __forceinline__ float dot4(float4 a) { return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, a.w * a.w))); }
template <typename T>
__device__ __forceinline__ void store_row4(T* p, float4 v);
template <>
__device__ __forceinline__ void store_row4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <>
__device__ __forceinline__ void store_row4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

// The pair of row r's token: its row of the table.  Thread 0 of the CTA that owns a portion's first row reads the previous token and
// leaves the portion's last one in its place.
__device__ __forceinline__ const uint16_t* pair_row(const RowParams& p, int r, long long* s_row) {
  const pi_token_pairs& k = p.pairs;
  if (threadIdx.x == 0) {
    const int seq = k.row_seq[r], row0 = k.seq_row0[seq];
    long long at = k.buckets;
    uint32_t* kept = reinterpret_cast<uint32_t*>(k.state + (size_t)k.slot[seq] * k.state_stride);
    if (r > row0 || k.seq_start[seq] > 0) {
      const uint32_t prev = r > row0 ? p.tokens[r - 1] : *kept;
      at = ((long long)prev * k.mul_prev + (long long)p.tokens[r] * k.mul_cur) % k.buckets;
    }
    if (r == row0) *kept = p.tokens[row0 + k.seq_n[seq] - 1];
    *s_row = at;
  }
  __syncthreads();
  return k.table + (size_t)*s_row * k.ld;
}
__device__ __forceinline__ float4 widen4(const uint16_t* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}

// HOLD: groups of four channels per thread, 0: any width, through shared memory one channel at a time.
template <typename T, RowSource SRC, int HOLD>
__global__ void __launch_bounds__(kRowThreads) row_rms_kernel(const RowParams p) {
  constexpr bool POST = SRC == kFromExperts || SRC == kFromResult;
  extern __shared__ __align__(16) float row[];
  __shared__ float red[2][kRowThreads / 32];
  __shared__ float s_w[64];
  __shared__ int s_at[64];
  const int r = blockIdx.x, tid = threadIdx.x;
  const int src = p.pick ? p.pick[r] : r;
  const pi_expert_sum& e = p.e;
  float4 wp[HOLD > 0 ? HOLD : 1];           // constants: ahead of the dependency wait
  if (POST && HOLD > 0) {
#pragma unroll
    for (int j = 0; j < HOLD; ++j) wp[j] = __ldg(reinterpret_cast<const float4*>(p.post_w + min((tid + j * kRowThreads) * 4, p.width - 4)));
  }
  if (SRC == kFromEmbedding) pi_grid_dependency_wait_strict();   // the step's fence, see pi_seq_batch
  else pi_grid_dependency_wait();
  float* x = p.x + (size_t)src * p.width;
  const uint16_t* t = SRC == kFromEmbedding ? p.table + (size_t)(p.tokens[r] % (uint32_t)p.vocab) * p.table_ld : nullptr;
  __shared__ long long s_pair;
  const uint16_t* pair = SRC == kFromEmbedding && p.pairs.table ? pair_row(p, r, &s_pair) : nullptr;
  const float* gate = POST && p.gate ? p.gate + (size_t)r * p.gate_stride : nullptr;
  if (SRC == kFromExperts) {
    if (tid < e.top) {
      s_w[tid] = e.weights[(size_t)r * e.top + tid];
      s_at[tid] = e.place ? e.place[(size_t)r * e.top + tid] : r * e.top + tid;
    }
    __syncthreads();
  }
  const float shared_gate = SRC == kFromExperts && e.shared_gate ? pi_sigmoid(e.shared_gate[(size_t)r * e.shared_gate_stride]) : 1.f;
  T* h = static_cast<T*>(p.h) + (size_t)r * p.ld_h;
  if (HOLD > 0) {
    float4 v[HOLD > 0 ? HOLD : 1];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < HOLD; ++j) {         // past the end: the last channels again, not counted
      const int i = (tid + j * kRowThreads) * 4, at = min(i, p.width - 4);
      if (SRC == kFromEmbedding) {
        v[j] = fma4(p.embed_scale, widen4(t + at), pair ? widen4(pair + at) : make_float4(0.f, 0.f, 0.f, 0.f));
      } else {
        v[j] = *reinterpret_cast<const float4*>(x + at);
      }
    }
    if (POST) {
      float4 y[HOLD > 0 ? HOLD : 1];
#pragma unroll
      for (int j = 0; j < HOLD; ++j) {
        const int i = (tid + j * kRowThreads) * 4, at = min(i, p.width - 4);
        if (SRC == kFromResult) {
          y[j] = *reinterpret_cast<const float4*>(p.y + (size_t)r * p.y_stride + at);
        } else {
          y[j] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (e.shared) y[j] = fma4(shared_gate, *reinterpret_cast<const float4*>(e.shared + (size_t)r * e.shared_stride + at), y[j]);
          for (int k0 = 0; k0 < e.top; k0 += 4) {
            float4 z[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) z[k] = expert_value4(e, (size_t)s_at[min(k0 + k, e.top - 1)] * e.y_stride + at);
#pragma unroll
            for (int k = 0; k < 4; ++k)
              if (k0 + k < e.top) y[j] = fma4(s_w[k0 + k], z[k], y[j]);
          }
        }
        if (gate) {
          const float4 z = *reinterpret_cast<const float4*>(gate + at), b = __ldg(reinterpret_cast<const float4*>(p.gate_bias + at));
          y[j] = make_float4(y[j].x * pi_sigmoid(z.x + b.x), y[j].y * pi_sigmoid(z.y + b.y), y[j].z * pi_sigmoid(z.z + b.z), y[j].w * pi_sigmoid(z.w + b.w));
        }
        if (p.of_sum) y[j] = fma4(p.keep, v[j], y[j]);
        if (i < p.width) ss += dot4(y[j]);
      }
      const float inv = 1.0f / sqrtf(row_sum_once(ss, red[0]) / (float)p.width + p.post_eps);
#pragma unroll
      for (int j = 0; j < HOLD; ++j) {
        if (p.of_sum) v[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        v[j] = make_float4(fmaf(y[j].x * inv, wp[j].x, v[j].x), fmaf(y[j].y * inv, wp[j].y, v[j].y), fmaf(y[j].z * inv, wp[j].z, v[j].z),
                           fmaf(y[j].w * inv, wp[j].w, v[j].w));
      }
    }
    ss = 0.f;
#pragma unroll
    for (int j = 0; j < HOLD; ++j) {
      const int i = (tid + j * kRowThreads) * 4;
      if (i >= p.width) continue;
      if (SRC != kFromX) *reinterpret_cast<float4*>(x + i) = v[j];
      ss += dot4(v[j]);
    }
    if (!p.h) return;
    const float inv = p.w ? 1.0f / sqrtf(row_sum_once(ss, red[1]) / (float)p.width + p.eps) : 1.f;
#pragma unroll
    for (int j = 0; j < HOLD; ++j) {
      const int i = (tid + j * kRowThreads) * 4;
      if (i >= p.width) continue;
      const float4 w = p.w ? __ldg(reinterpret_cast<const float4*>(p.w + i)) : make_float4(1.f, 1.f, 1.f, 1.f);
      store_row4<T>(h + i, make_float4(v[j].x * inv * w.x, v[j].y * inv * w.y, v[j].z * inv * w.z, v[j].w * inv * w.w));
    }
    return;
  }
  float ss = 0.f;
  if (POST) {
    for (int i = tid; i < p.width; i += kRowThreads) {
      float v = 0.f;
      if (SRC == kFromResult) {
        v = p.y[(size_t)r * p.y_stride + i];
      } else {
        if (e.shared) v = shared_gate * e.shared[(size_t)r * e.shared_stride + i];
        for (int k = 0; k < e.top; ++k) v = fmaf(s_w[k], expert_value(e, (size_t)s_at[k] * e.y_stride + i), v);
      }
      if (gate) v *= pi_sigmoid(gate[i] + __ldg(p.gate_bias + i));
      if (p.of_sum) v = fmaf(p.keep, x[i], v);
      row[i] = v;
      ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(row_sum_once(ss, red[0]) / (float)p.width + p.post_eps);
    ss = 0.f;
    for (int i = tid; i < p.width; i += kRowThreads) {   // every thread its own channels, as above
      const float v = fmaf(row[i] * inv, __ldg(p.post_w + i), p.of_sum ? 0.f : x[i]);
      x[i] = v;
      row[i] = v;
      ss = fmaf(v, v, ss);
    }
  } else {
    for (int i = tid; i < p.width; i += kRowThreads) {
      const float v = SRC == kFromEmbedding ? fmaf(p.embed_scale, pi_bf16_bits_to_f32(t[i]), pair ? pi_bf16_bits_to_f32(pair[i]) : 0.f) : x[i];
      if (SRC == kFromEmbedding) x[i] = v;
      row[i] = v;
      ss = fmaf(v, v, ss);
    }
  }
  if (!p.h) return;
  const float inv = p.w ? 1.0f / sqrtf(row_sum_once(ss, red[1]) / (float)p.width + p.eps) : 1.f;
  for (int i = tid; i < p.width; i += kRowThreads) h[i] = pi_from_f32<T>(p.w ? row[i] * inv * __ldg(p.w + i) : row[i]);
}

template <typename T, int HOLD>
void (*pick_rms(RowSource s))(const RowParams) {
  return s == kFromX ? row_rms_kernel<T, kFromX, HOLD> : s == kFromEmbedding ? row_rms_kernel<T, kFromEmbedding, HOLD>
         : s == kFromExperts ? row_rms_kernel<T, kFromExperts, HOLD> : row_rms_kernel<T, kFromResult, HOLD>;
}
template <typename T>
void (*pick_rms(RowSource s, const RowParams& p, bool in_registers))(const RowParams) {
  if (!in_registers) return pick_rms<T, 0>(s);
  return p.width <= 4 * kRowThreads ? pick_rms<T, 1>(s) : p.width <= 8 * kRowThreads ? pick_rms<T, 2>(s) : pick_rms<T, 4>(s);
}

}  // namespace

pi_status pi_launch_row_norm(pi_ctx* ctx, const pi_row_norm& n) {
  pi_prof_scope prof(ctx, PI_PROF_OTHER);
  RowParams p = {n.x, n.width, n.pick, n.table, n.table_ld, n.vocab, n.tokens, {}, n.norm.w, n.norm.eps, n.h, n.ld_h,
                 n.y, n.y_stride, n.post.w, n.post.eps, n.embed_scale, n.of_sum, n.keep, n.gate, n.gate_bias, n.gate_stride, n.pairs};
  if (n.experts) p.e = *n.experts;
  PI_REQUIRE(ctx, p.e.top <= 64, "at most 64 experts per token, not %d", p.e.top);
  const bool bf16 = n.h_kind == PI_BF16;
  void (*k)(const RowParams);
  bool in_registers = false;
  if (n.rms) {
    PI_REQUIRE(ctx, !(n.y || n.experts) || n.post.w, "a sublayer's result needs its norm");
    const RowSource src = n.table ? kFromEmbedding : n.experts ? kFromExperts : n.y ? kFromResult : kFromX;
    const bool aligned = n.width % 4 == 0 && n.ld_h % 4 == 0 && (!n.table || n.table_ld % 4 == 0) && (!n.y || n.y_stride % 4 == 0) &&
                         (!n.experts || (p.e.y_stride % 4 == 0 && p.e.shared_stride % 4 == 0 && !p.e.scale)) &&
                         (!n.gate || (n.gate_stride % 4 == 0 && (uintptr_t)n.gate % 16 == 0)) && (!n.pairs.table || n.pairs.ld % 4 == 0);
    PI_REQUIRE(ctx, !n.experts || !p.e.scale, "a scale per channel belongs to layer norm");
    PI_REQUIRE(ctx, !n.gate || n.gate_bias, "a gate needs its bias");
    in_registers = aligned && n.width <= 16 * kRowThreads;
    k = bf16 ? pick_rms<__nv_bfloat16>(src, p, in_registers) : pick_rms<float>(src, p, in_registers);
  } else if (n.of_sum || n.gate || n.pairs.table) {
    return pi_fail(ctx, PI_ERR_INVALID_ARG, "norms of the sum, gates and token pairs belong to RMS norms");
  } else if (n.table) k = bf16 ? row_norm_kernel<__nv_bfloat16, kFromEmbedding> : row_norm_kernel<float, kFromEmbedding>;
  else if (n.experts) k = bf16 ? row_norm_kernel<__nv_bfloat16, kFromExperts> : row_norm_kernel<float, kFromExperts>;
  else k = bf16 ? row_norm_kernel<__nv_bfloat16, kFromX> : row_norm_kernel<float, kFromX>;
  const size_t smem = in_registers ? 0 : (size_t)n.width * sizeof(float);
  PI_REQUIRE(ctx, smem <= kSmemFit, "rows of %d channels are too wide", n.width);
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(n.rows), dim3(kRowThreads), smem, 1, p));
  return PI_OK;
}
