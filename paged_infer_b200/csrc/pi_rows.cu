// Row-wise steps of designs whose sublayers are normalised before (layer norm: zero mean, unit variance, a weight, no bias):
// one CTA per row takes up what the last sublayer left - the embedding, the residual row as it is, or the outputs of the
// row's experts - and writes the next sublayer's input.  All sums are f32; mean and variance are two passes over the row in
// shared memory.
#include <algorithm>

#include "pi_layered.cuh"

namespace {

constexpr int kRowThreads = 256;

enum RowSource { kFromX, kFromEmbedding, kFromExperts };

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

}  // namespace

pi_status pi_launch_row_norm(pi_ctx* ctx, const pi_row_norm& n) {
  pi_prof_scope prof(ctx, PI_PROF_OTHER);
  RowParams p = {n.x, n.width, n.pick, n.table, n.table_ld, n.vocab, n.tokens, {}, n.norm.w, n.norm.eps, n.h, n.ld_h};
  if (n.experts) p.e = *n.experts;
  PI_REQUIRE(ctx, p.e.top <= 64, "at most 64 experts per token, not %d", p.e.top);
  const bool bf16 = n.h_kind == PI_BF16;
  void (*k)(const RowParams);
  if (n.table) k = bf16 ? row_norm_kernel<__nv_bfloat16, kFromEmbedding> : row_norm_kernel<float, kFromEmbedding>;
  else if (n.experts) k = bf16 ? row_norm_kernel<__nv_bfloat16, kFromExperts> : row_norm_kernel<float, kFromExperts>;
  else k = bf16 ? row_norm_kernel<__nv_bfloat16, kFromX> : row_norm_kernel<float, kFromX>;
  const size_t smem = (size_t)n.width * sizeof(float);
  PI_REQUIRE(ctx, smem <= 48 * 1024, "rows of %d channels are too wide", n.width);
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(n.rows), dim3(kRowThreads), smem, 1, p));
  return PI_OK;
}
