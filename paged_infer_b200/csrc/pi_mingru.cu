// minGRU: a gated recurrence of single channels whose gates read only the current token, f32 throughout:
//
//   z = sigmoid(zl + bz),  u = ul + bx,  c = u + 1/2 (u >= 0) or sigmoid(u)
//   S_t = (1 - z) S_(t-1) + z c,   out = S_t silu(g)
//
// mingru_scan_kernel: a thread per channel (or four adjacent ones) walks the tokens of a sequence, a batch of loads ahead of the
// arithmetic; the decode kernel, and the one of short portions and the f32 mode.
// mingru_stream_kernel: long portions.  A step is the map S -> a S + b, and maps compose.  A CTA owns 32 channels of a sequence and
// streams their operands through a ring of asynchronous copies, kPass tokens at a time; every warp holds the maps of a segment of
// them and publishes its composition, so that what enters a segment is a short fold over the segments before it.  Every operand is
// read once, and the next passes are in flight meanwhile.  1 - z is formed without cancellation; all factors lie in [0, 1], so no
// product overflows.
// The arithmetic per element counts here (three sigmoids each): exponentials and reciprocals are the hardware's, a few units in the
// last place.
#include <algorithm>

#include "pi_layered.cuh"
#include "pi_mma.cuh"

namespace {

constexpr int kScanThreads = 64, kScanAhead = 4;
constexpr int kWarps = 16, kLen = 8, kPass = kWarps * kLen, kStages = 4;   // tokens of a segment, of a pass; passes in shared memory
constexpr size_t kStreamSmem = (size_t)kStages * 3 * kPass * 32 * sizeof(float);

struct GruParams {
  pi_mingru r;
  const float* proj;
  size_t stride;
  void* out;
  size_t out_stride;
  const int32_t *seqs, *seq_row0, *seq_n, *seq_start, *slot;
};

// V adjacent channels.
template <int V>
struct Floats {
  float v[V];
};
template <int V>
__device__ __forceinline__ Floats<V> load(const float* p) {
  Floats<V> r;
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    r.v[0] = f.x;
    r.v[1] = f.y;
    r.v[2] = f.z;
    r.v[3] = f.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int V>
__device__ __forceinline__ void store(float* p, const Floats<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int V>
__device__ __forceinline__ void store(__nv_bfloat16* p, const Floats<V>& r) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    *p = __float2bfloat16_rn(r.v[0]);
  }
}

__device__ __forceinline__ float gru_sigmoid(float x) {
  const float e = __expf(-fabsf(x)), inv = __fdividef(1.0f, 1.0f + e);
  return x >= 0.f ? inv : e * inv;
}
// One step as a map: S -> a S + b.
struct GruStep {
  float a, b;
};
__device__ __forceinline__ GruStep gru_step(float zl, float ul) {
  const float e = __expf(-fabsf(zl)), inv = __fdividef(1.0f, 1.0f + e), small = e * inv;
  const float c = ul >= 0.f ? ul + 0.5f : gru_sigmoid(ul);
  return zl >= 0.f ? GruStep{small, inv * c} : GruStep{inv, small * c};
}
__device__ __forceinline__ GruStep then(GruStep first, GruStep second) { return {first.a * second.a, fmaf(second.a, first.b, second.b)}; }

template <typename O, int V>
__global__ void __launch_bounds__(kScanThreads) mingru_scan_kernel(const GruParams p) {
  const pi_mingru& r = p.r;
  const int seq = p.seqs[blockIdx.y], c = (blockIdx.x * kScanThreads + threadIdx.x) * V;
  const int row0 = p.seq_row0[seq], n = p.seq_n[seq];
  const bool is = c < r.width;                       // V > 1: the width is a multiple of V
  float* st = r.state + (size_t)p.slot[seq] * r.state_stride + r.state_off + (is ? c : 0);
  // the state was written by an earlier step: it may be read ahead of the dependency wait
  Floats<V> S = load<V>(st), bz = load<V>(r.z_bias + (is ? c : 0)), bx = load<V>(r.x_bias + (is ? c : 0));
  if (p.seq_start[seq] == 0) {
#pragma unroll
    for (int k = 0; k < V; ++k) S.v[k] = 0.f;
  }
  pi_grid_dependency_wait();
  if (!is) return;
  const float* x = p.proj + (size_t)row0 * p.stride + c;
  O* o = static_cast<O*>(p.out) + (size_t)row0 * p.out_stride + c;
  for (int t0 = 0; t0 < n; t0 += kScanAhead) {
    Floats<V> z[kScanAhead], u[kScanAhead], g[kScanAhead];
#pragma unroll
    for (int j = 0; j < kScanAhead; ++j) {
      if (j > 0 && t0 + j >= n) break;
      const float* xt = x + (size_t)(t0 + j) * p.stride;
      z[j] = load<V>(xt + r.col_z);
      u[j] = load<V>(xt + r.col_x);
      g[j] = load<V>(xt + r.col_g);
    }
#pragma unroll
    for (int j = 0; j < kScanAhead; ++j) {
      if (j > 0 && t0 + j >= n) break;
      Floats<V> y;
#pragma unroll
      for (int k = 0; k < V; ++k) {
        const GruStep s = gru_step(z[j].v[k] + bz.v[k], u[j].v[k] + bx.v[k]);
        S.v[k] = fmaf(s.a, S.v[k], s.b);
        y.v[k] = S.v[k] * g[j].v[k] * gru_sigmoid(g[j].v[k]);
      }
      store<V>(o + (size_t)(t0 + j) * p.out_stride, y);
    }
  }
  store<V>(st, S);
}

// A lane holds one channel.  V: channels of an asynchronous copy, 4 or 1.
template <typename O, int V>
__global__ void __launch_bounds__(kWarps * 32) mingru_stream_kernel(const GruParams p) {
  extern __shared__ __align__(16) float ring[];       // [stage][z, u, g][token][32]
  __shared__ GruStep seg[kWarps][32];
  const pi_mingru& r = p.r;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = p.seqs[blockIdx.y], c0 = blockIdx.x * 32, c = c0 + lane;
  const int row0 = p.seq_row0[seq], n = p.seq_n[seq];
  const bool is = c < r.width;
  float* st = r.state + (size_t)p.slot[seq] * r.state_stride + r.state_off + (is ? c : 0);
  float S = p.seq_start[seq] != 0 ? *st : 0.f;         // written by an earlier step, as in the scan
  const float bz = __ldg(r.z_bias + (is ? c : 0)), bx = __ldg(r.x_bias + (is ? c : 0));
  pi_grid_dependency_wait();
  auto fetch = [&](int pass) {
    const int base = pass * kPass, count = min(kPass, n - base);   // <= 0 behind the last pass: nothing
    float* dst = ring + (size_t)(pass % kStages) * 3 * kPass * 32;
    const float* src = p.proj + (size_t)(row0 + base) * p.stride + c0;
    for (int i = tid; i < count * (32 / V); i += kWarps * 32) {
      const int t = i / (32 / V), x = (i - t * (32 / V)) * V;
      const bool ok = c0 + x < r.width;
#pragma unroll
      for (int k = 0; k < 3; ++k) {
        const float* from = ok ? src + (size_t)t * p.stride + (k == 0 ? r.col_z : k == 1 ? r.col_x : r.col_g) + x : p.proj;
        const uint32_t to = pi_mma::smem_addr(dst + (k * kPass + t) * 32 + x);
        if constexpr (V == 4) pi_mma::cp_async16(to, from, ok ? 16 : 0);
        else asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(to), "l"(from), "r"(ok ? 4 : 0) : "memory");
      }
    }
    pi_mma::cp_async_commit();
  };
  for (int s = 0; s < kStages - 1; ++s) fetch(s);
  for (int pass = 0; pass * kPass < n; ++pass) {
    pi_mma::cp_async_wait<kStages - 2>();
    __syncthreads();                                   // this pass has landed, and the last one's stage and segments are free
    fetch(pass + kStages - 1);
    const int left = min(kPass, n - pass * kPass), len = (left + kWarps - 1) / kWarps, t0 = warp * len, mine = min(len, left - t0);
    const float* x = ring + (size_t)(pass % kStages) * 3 * kPass * 32 + lane;
    GruStep m[kLen], all = {1.f, 0.f};
    float g[kLen];
#pragma unroll
    for (int j = 0; j < kLen; ++j) {
      m[j] = {1.f, 0.f};
      if (j < mine) {
        const float* xt = x + (t0 + j) * 32;
        m[j] = gru_step(xt[0] + bz, xt[kPass * 32] + bx);
        const float z = xt[2 * kPass * 32];
        g[j] = z * gru_sigmoid(z);
      }
    }
#pragma unroll
    for (int j = 0; j < kLen; ++j) all = then(all, m[j]);
    seg[warp][lane] = all;
    __syncthreads();
    float in = S;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const GruStep s = seg[w][lane];
      if (w == warp) in = S;
      S = fmaf(s.a, S, s.b);
    }
    if (is) {
      O* o = static_cast<O*>(p.out) + (size_t)(row0 + pass * kPass + t0) * p.out_stride + c;
#pragma unroll
      for (int j = 0; j < kLen; ++j) {
        in = fmaf(m[j].a, in, m[j].b);
        if (j < mine) o[(size_t)j * p.out_stride] = pi_from_f32<O>(in * g[j]);
      }
    }
  }
  pi_mma::cp_async_wait<0>();
  if (is && warp == 0) *st = S;
}

template <typename O, int V>
cudaError_t grant(pi_ctx* ctx) {
  static pi_smem_grant granted;
  if (granted.of(ctx) >= kStreamSmem) return cudaSuccess;
  granted.of(ctx) = kStreamSmem;
  return cudaFuncSetAttribute(mingru_stream_kernel<O, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kStreamSmem);
}

template <typename O, int V>
pi_status stream(pi_ctx* ctx, const GruParams& p, int n_seqs) {
  PI_CUDA(ctx, (grant<O, V>(ctx)));
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, mingru_stream_kernel<O, V>, dim3((p.r.width + 31) / 32, n_seqs), dim3(kWarps * 32), kStreamSmem, 1, p));
  return PI_OK;
}

}  // namespace

pi_status pi_launch_mingru(pi_ctx* ctx, const pi_mingru& r, const float* proj, size_t stride, void* out, size_t out_stride, int out_kind,
                           const pi_seq_batch& b) {
  pi_prof_scope prof(ctx, PI_PROF_RECURRENCE);
  GruParams p = {r, proj, stride, out, out_stride, b.scan_seqs, b.seq_row0, b.seq_n, b.seq_start, b.slot};
  auto even = [&](int v) {
    return r.width % v == 0 && r.col_z % v == 0 && r.col_x % v == 0 && r.col_g % v == 0 && stride % v == 0 && out_stride % v == 0 && r.state_off % v == 0 &&
           r.state_stride % v == 0;
  };
  const bool bf16 = out_kind == PI_BF16;
  if (b.n_scan > 0) {
    const int v = even(4) ? 4 : 1;
    auto k = v == 4 ? (bf16 ? mingru_scan_kernel<__nv_bfloat16, 4> : mingru_scan_kernel<float, 4>)
                    : (bf16 ? mingru_scan_kernel<__nv_bfloat16, 1> : mingru_scan_kernel<float, 1>);
    const int per_cta = kScanThreads * v;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3((r.width + per_cta - 1) / per_cta, b.n_scan), dim3(kScanThreads), 0, 1, p));
  }
  if (b.n_chunk_seqs > 0) {
    p.seqs = b.chunk_seqs;
    const bool vec = even(4) && (uintptr_t)proj % 16 == 0;
    if (bf16) return vec ? stream<__nv_bfloat16, 4>(ctx, p, b.n_chunk_seqs) : stream<__nv_bfloat16, 1>(ctx, p, b.n_chunk_seqs);
    return vec ? stream<float, 4>(ctx, p, b.n_chunk_seqs) : stream<float, 1>(ctx, p, b.n_chunk_seqs);
  }
  return PI_OK;
}
