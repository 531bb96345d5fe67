// Recurrences with a scalar decay per head, f32 throughout.  State space (Mamba-2):
//
//   u_t = silu(b + sum_j w_j (x, B, C)_(t - taps + 1 + j))       per channel, zeros before the start
//   dt  = softplus(dt_t + bias),  a = exp(-exp(A_log) dt)         per head
//   S_t = a S_(t-1) + dt B_t x_t^T,   y_t = (S_t^T C_t + D x_t) silu(z_t)
//   out = y / rms(y) * norm                                       over each of norm_groups equal parts of all heads together
//
// B and C are common to the heads of a group.  Lightning attention is the same with a constant decay, dt = 1, no convolution and no
// D, a group per head (B: keys, C: queries, x: values) and the gate behind the norm:
//
//   u_t = silu(x, B, C);  S_t = decay S_(t-1) + B_t x_t^T,   y_t = S_t^T C_t,   out = y / rms(y) * norm * sigmoid(z)
//
// ssd_scan_kernel walks the tokens of a sequence with the state in registers (decoding, short portions, f32): CTA = (128 value
// columns of a head, sequence); a thread holds four columns of every (256 / lanes per row)-th state channel.  The
// convolution runs inside it; its last inputs move on in the next kernel, when every head has read them.  For state sizes
// that do not fit the registers the state stays in global memory (R = 0).  Long portions take pi_ssd_chunk.cu.
// ssd_norm_kernel normalises y and moves the convolution's inputs on.
#include <math.h>

#include <algorithm>

#include "pi_layered.cuh"

namespace {

constexpr int kThreads = 256, kWarps = 8, kSlice = 128;

struct ScanParams {
  pi_ssd r;
  const float* proj;
  size_t stride;
  float* y;
  const int32_t *seqs, *seq_row0, *seq_n, *seq_start, *slot;
  int lanes_log2;      // lanes per state row: a power of two
  int vec;
};

__device__ __forceinline__ float silu(float v) { return v * pi_sigmoid(v); }

// ITEMS: channels of the convolution per thread.
template <int R, int ITEMS>
__global__ void __launch_bounds__(kThreads, R == 0 || R > 16 ? 1 : R > 8 || ITEMS > 2 ? 2 : 4) ssd_scan_kernel(const ScanParams p) {
  extern __shared__ __align__(16) float sm[];
  const pi_ssd& r = p.r;
  const int e_first = blockIdx.x * kSlice, head = blockIdx.y, seq = p.seqs[blockIdx.z];
  const int cols = min(kSlice, r.vdim - e_first), N = r.dim, group = head / (r.heads / r.groups), inner = r.inner(), channels = r.channels();
  float* sx = sm;                          // [kSlice] x, [N] B, [N] C behind the convolution
  float* sB = sx + kSlice;
  float* sC = sB + N;
  __shared__ __align__(16) float part[kWarps][kSlice];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int row0 = p.seq_row0[seq], n_tok = p.seq_n[seq];
  const bool fresh = p.seq_start[seq] == 0;
  const int lpr = 1 << p.lanes_log2, c4 = (tid & (lpr - 1)) * 4, r_first = tid >> p.lanes_log2, rpp = kThreads >> p.lanes_log2;
  const int nv = min(4, cols - c4);        // columns of this thread that exist (may be <= 0)
  float* slot = r.state + (size_t)p.slot[seq] * r.state_stride + r.state_off;
  float* S = slot + ((size_t)head * N) * r.vdim + e_first + c4;
  const float* past = slot + (size_t)r.heads * N * r.vdim;   // [taps - 1][channels]
  const float a_neg = r.decay ? 0.f : -expf(__ldg(r.a_log + head)), dt_bias = r.decay ? 0.f : __ldg(r.dt_bias + head), skip = r.d ? __ldg(r.d + head) : 0.f;
  const float fixed = r.decay ? __ldg(r.decay + head) : 0.f;

  auto load4 = [&](const float* src) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.vec) {
      if (nv > 0) v = *reinterpret_cast<const float4*>(src);
    } else {
      if (nv > 0) v.x = src[0];
      if (nv > 1) v.y = src[1];
      if (nv > 2) v.z = src[2];
      if (nv > 3) v.w = src[3];
    }
    return v;
  };
  auto store4 = [&](float* dst, float4 v) {
    if (p.vec) {
      if (nv > 0) *reinterpret_cast<float4*>(dst) = v;
    } else {
      if (nv > 0) dst[0] = v.x;
      if (nv > 1) dst[1] = v.y;
      if (nv > 2) dst[2] = v.z;
      if (nv > 3) dst[3] = v.w;
    }
  };
  // item i of this CTA's channels: its channel among x, B, C, and its place in shared memory
  const int items = cols + 2 * N;
  auto channel = [&](int i) {
    if (i < cols) return head * r.vdim + e_first + i;
    i -= cols;
    return i < N ? inner + group * N + i : inner + r.groups * N + group * N + (i - N);
  };
  for (int i = cols + tid; i < kSlice; i += kThreads) sx[i] = 0.f;

  // what earlier steps left may be read ahead of the dependency wait
  float4 s[R > 0 ? R : 1];
  if (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int n = r_first + i * rpp;
      s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && n < N) s[i] = load4(S + (size_t)n * r.vdim);
    }
  }
  float hist[ITEMS][3];                    // up to four taps: the channel's last three inputs
  if (r.conv4) {
#pragma unroll
    for (int q = 0; q < ITEMS; ++q) {
      const int i = tid + q * kThreads, c = i < items ? channel(i) : 0;
#pragma unroll
      for (int j = 0; j < 3; ++j) {
        const int back = r.taps - 4 + j;   // place among the inputs kept; below 0: a tap there is not
        hist[q][j] = !fresh && i < items && back >= 0 ? past[(size_t)back * channels + c] : 0.f;
      }
    }
  }
  pi_grid_dependency_wait();

  for (int t = 0; t < n_tok; ++t) {
    const float* x = p.proj + (size_t)(row0 + t) * p.stride;
    __syncthreads();                       // the last token's channels and partial sums have been read
    if (r.conv4) {
      float u[ITEMS];
      float4 w[ITEMS];
#pragma unroll
      for (int q = 0; q < ITEMS; ++q) {
        const int i = tid + q * kThreads, c = channel(min(i, items - 1));
        u[q] = x[r.col_x + c];
        w[q] = __ldg(r.conv4 + c);
      }
#pragma unroll
      for (int q = 0; q < ITEMS; ++q) {
        const int i = tid + q * kThreads;
        const float v = fmaf(w[q].w, u[q], fmaf(w[q].z, hist[q][2], fmaf(w[q].y, hist[q][1], fmaf(w[q].x, hist[q][0], __ldg(r.conv_b + channel(min(i, items - 1)))))));
        hist[q][0] = hist[q][1];
        hist[q][1] = hist[q][2];
        hist[q][2] = u[q];
        if (i < items) sm[i < cols ? i : i - cols + kSlice] = silu(v);
      }
    } else if (!r.conv) {
      float u[ITEMS];
#pragma unroll
      for (int q = 0; q < ITEMS; ++q) u[q] = x[r.col_x + channel(min(tid + q * kThreads, items - 1))];
#pragma unroll
      for (int q = 0; q < ITEMS; ++q) {
        const int i = tid + q * kThreads;
        if (i < items) sm[i < cols ? i : i - cols + kSlice] = silu(u[q]);
      }
    } else {
      for (int i = tid; i < items; i += kThreads) {
        const int c = channel(i);
        float v = __ldg(r.conv_b + c);
        for (int j = 0; j < r.taps; ++j) {
          const int tt = t - r.taps + 1 + j;
          const float u = tt >= 0 ? p.proj[(size_t)(row0 + tt) * p.stride + r.col_x + c] : fresh ? 0.f : past[(size_t)(r.taps - 1 + tt) * channels + c];
          v = fmaf(__ldg(r.conv + (size_t)c * r.taps + j), u, v);
        }
        sm[i < cols ? i : i - cols + kSlice] = silu(v);
      }
    }
    const float dt = r.decay ? 1.f : pi_softplus(x[r.col_dt + head] + dt_bias), keep = r.decay ? fixed : expf(a_neg * dt);
    __syncthreads();
    float4 xv = *reinterpret_cast<const float4*>(sx + c4);
    xv = make_float4(dt * xv.x, dt * xv.y, dt * xv.z, dt * xv.w);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    auto step = [&](float4& sv, int n) {
      const float b = sB[n], c = sC[n];
      sv.x = fmaf(keep, sv.x, b * xv.x);
      sv.y = fmaf(keep, sv.y, b * xv.y);
      sv.z = fmaf(keep, sv.z, b * xv.z);
      sv.w = fmaf(keep, sv.w, b * xv.w);
      o.x = fmaf(sv.x, c, o.x);
      o.y = fmaf(sv.y, c, o.y);
      o.z = fmaf(sv.z, c, o.z);
      o.w = fmaf(sv.w, c, o.w);
    };
    if (R > 0) {
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int n = r_first + i * rpp;
        if (n < N) step(s[i], n);
      }
    } else {
      for (int n = r_first; n < N; n += rpp) {
        float4 sv = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!(fresh && t == 0)) sv = load4(S + (size_t)n * r.vdim);
        step(sv, n);
        store4(S + (size_t)n * r.vdim, sv);
      }
    }
    for (int k = lpr; k < 32; k <<= 1) {   // rows that share a warp
      o.x += __shfl_xor_sync(0xffffffffu, o.x, k);
      o.y += __shfl_xor_sync(0xffffffffu, o.y, k);
      o.z += __shfl_xor_sync(0xffffffffu, o.z, k);
      o.w += __shfl_xor_sync(0xffffffffu, o.w, k);
    }
    if (lane < lpr) *reinterpret_cast<float4*>(&part[warp][c4]) = o;
    __syncthreads();
    if (tid < cols) {
      float v = skip * sx[tid];
#pragma unroll
      for (int w = 0; w < kWarps; ++w) v += part[w][tid];
      const int e = head * r.vdim + e_first + tid;
      p.y[(size_t)(row0 + t) * inner + e] = r.gate_last ? v : v * silu(x[r.col_z + e]);
    }
  }
  if (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int n = r_first + i * rpp;
      if (n < N) store4(S + (size_t)n * r.vdim, s[i]);
    }
  }
}

struct NormParams {
  pi_ssd r;
  const float* proj;
  size_t stride;
  const float* y;
  void* out;
  size_t out_stride;
  int rows;
  const int32_t *seq_row0, *seq_n, *seq_start, *slot;
};

// blockIdx.x < rows: (row, part of the channels); behind them: 256 of the convolution's channels of a sequence.
constexpr int kHeld = 4;                   // groups of four channels a thread keeps between the two passes
template <typename O>
__global__ void __launch_bounds__(kThreads) ssd_norm_kernel(const NormParams p) {
  const pi_ssd& r = p.r;
  const int tid = threadIdx.x, inner = r.inner();
  __shared__ float red[kWarps];
  pi_grid_dependency_wait();
  if ((int)blockIdx.x >= p.rows) {
    const int channels = r.channels(), blocks = (channels + kThreads - 1) / kThreads, i = (int)blockIdx.x - p.rows, seq = i / blocks;
    const int n = p.seq_n[seq], keep = r.taps - 1, c = (i - seq * blocks) * kThreads + tid;
    if (blockIdx.y > 0 || c >= channels) return;
    const bool fresh = p.seq_start[seq] == 0;
    float* past = r.state + (size_t)p.slot[seq] * r.state_stride + r.state_off + (size_t)r.heads * r.dim * r.vdim + c;
    const float* x = p.proj + (size_t)p.seq_row0[seq] * p.stride + r.col_x + c;
    auto input = [&](int j) {                // what stands at place j from now on
      const int t = n - keep + j;
      return t >= 0 ? x[(size_t)t * p.stride] : fresh ? 0.f : past[(size_t)(j + n) * channels];
    };
    if (keep <= 3) {
      float v[3];
#pragma unroll
      for (int j = 0; j < 3; ++j) v[j] = j < keep ? input(j) : 0.f;
#pragma unroll
      for (int j = 0; j < 3; ++j)
        if (j < keep) past[(size_t)j * channels] = v[j];
    } else {
      for (int j = 0; j < keep; ++j) past[(size_t)j * channels] = input(j);   // ascending: an input moves towards the front
    }
    return;
  }
  const int n = inner / r.norm_groups, c0 = blockIdx.y * n;
  const float* y = p.y + (size_t)blockIdx.x * inner + c0;
  const bool held = n % 4 == 0 && n <= kHeld * 4 * kThreads;
  float4 v[kHeld];
  float ss = 0.f;
  if (held) {
#pragma unroll
    for (int j = 0; j < kHeld; ++j) {
      const int i = (tid + j * kThreads) * 4;
      v[j] = *reinterpret_cast<const float4*>(y + min(i, n - 4));
      if (i < n) ss = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, fmaf(v[j].z, v[j].z, fmaf(v[j].w, v[j].w, ss))));
    }
  } else {
    for (int i = tid; i < n; i += kThreads) ss = fmaf(y[i], y[i], ss);
  }
  ss = pi_warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) ss += red[w];
  const float inv = 1.0f / sqrtf(ss / (float)n + r.eps);
  O* out = static_cast<O*>(p.out) + (size_t)blockIdx.x * p.out_stride + c0;
  const float* z = p.proj + (size_t)blockIdx.x * p.stride + r.col_z + c0;
  if (held) {
#pragma unroll
    for (int j = 0; j < kHeld; ++j) {
      const int i = (tid + j * kThreads) * 4;
      if (i >= n) break;
      const float e[4] = {v[j].x, v[j].y, v[j].z, v[j].w};
      float gate[4] = {1.f, 1.f, 1.f, 1.f};
      if (r.gate_last) {
#pragma unroll
        for (int k = 0; k < 4; ++k) gate[k] = pi_sigmoid(z[i + k]);
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) out[i + k] = pi_from_f32<O>(e[k] * inv * __ldg(r.norm + c0 + i + k) * gate[k]);
    }
  } else {
    for (int i = tid; i < n; i += kThreads) out[i] = pi_from_f32<O>(y[i] * inv * __ldg(r.norm + c0 + i) * (r.gate_last ? pi_sigmoid(z[i]) : 1.f));
  }
}

template <int ITEMS>
void (*pick_scan(int rows))(const ScanParams) {
  return rows <= 2 ? ssd_scan_kernel<2, ITEMS> : rows <= 4 ? ssd_scan_kernel<4, ITEMS> : rows <= 8 ? ssd_scan_kernel<8, ITEMS>
         : rows <= 16 ? ssd_scan_kernel<16, ITEMS> : rows <= 32 ? ssd_scan_kernel<32, ITEMS> : ssd_scan_kernel<0, ITEMS>;
}

}  // namespace

pi_status pi_launch_ssd(pi_ctx* ctx, const pi_ssd& r, const float* proj, size_t stride, float* y, void* out, size_t out_stride, int out_kind,
                        const pi_seq_batch& b, float* scratch) {
  pi_prof_scope prof(ctx, PI_PROF_RECURRENCE);
  if (b.n_scan > 0) {
    ScanParams p = {r, proj, stride, y, b.scan_seqs, b.seq_row0, b.seq_n, b.seq_start, b.slot, 0, 0};
    while ((4 << p.lanes_log2) < std::min(r.vdim, kSlice)) ++p.lanes_log2;
    p.vec = r.vdim % 4 == 0 && r.state_off % 4 == 0 && r.state_stride % 4 == 0;
    const int rpp = kThreads >> p.lanes_log2, need = (r.dim + rpp - 1) / rpp;
    const int items = (std::min(r.vdim, kSlice) + 2 * r.dim + kThreads - 1) / kThreads;   // per thread
    PI_REQUIRE(ctx, items <= 8, "%d state channels are too many", r.dim);
    void (*k)(const ScanParams) = items <= 2 ? pick_scan<2>(need) : items <= 4 ? pick_scan<4>(need) : pick_scan<8>(need);
    const size_t smem = (size_t)(kSlice + 2 * r.dim) * sizeof(float);
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3((r.vdim + kSlice - 1) / kSlice, r.heads, b.n_scan), dim3(kThreads), smem, 1, p));
  }
  if (b.n_chunks > 0) PI_TRY(pi_launch_ssd_chunks(ctx, r, proj, stride, y, b, scratch));
  const NormParams n = {r, proj, stride, y, out, out_stride, b.rows, b.seq_row0, b.seq_n, b.seq_start, b.slot};
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, out_kind == PI_BF16 ? ssd_norm_kernel<__nv_bfloat16> : ssd_norm_kernel<float>,
                                  dim3(b.rows + (r.taps > 1 ? b.n_seqs * ((r.channels() + kThreads - 1) / kThreads) : 0), r.norm_groups), dim3(kThreads), 0, 1, n));
  return PI_OK;
}
