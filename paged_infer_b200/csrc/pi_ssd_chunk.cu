// Portions of many tokens through the recurrence of pi_ssd.cu, in chunks of 64 tokens that run side by side.  With
// F_t = running sum of -exp(A_log) dt inside the chunk (never positive):
//
//   1. ssd_conv_kernel      convolution and silu of x, B, C; dt and F     (silu_planes_kernel: without a convolution)
//   2. ssd_local_kernel     what the chunk adds to the state: U = sum_s e^(F_end - F_s) dt_s B_s x_s^T
//   3. ssd_pass_kernel      the state in front of every chunk, one pass over the chunks (S <- e^F_end S + U); it takes U's place
//   4. ssd_output_kernel    y_t = e^(F_t) S^T C_t + sum_(s <= t) (C_t . B_s) e^(F_t - F_s) dt_s x_s + D x_t, times silu(z_t)
//
// The recurrence is f32: operands of the tensor-core products (mma.sync) are pairs of bf16 planes, hi + lo (16 bits), three
// products each.  The convolution leaves x, B and C as planes, padded to 16 channels and to whole chunks, so that the later
// kernels only copy; the pass leaves the state as packed pairs.  B and C are common to a group's heads: a CTA takes several
// heads of one group and scores C . B once for all of them.  (Lightning attention: no convolution, dt = 1, F = t ln(decay), no D; the
// gate follows with the norm.)
#include <math.h>

#include <algorithm>

#include "pi_layered.cuh"
#include "pi_mma.cuh"

namespace {
using namespace pi_mma;

constexpr int C = kRecurrenceChunk, kVS = 64;
constexpr int kThreads = 256, kWarps = 8;
constexpr int kMaxDim = 256;
constexpr int kMaxHeads = 4;             // heads of a CTA
constexpr int kApitch = C + 4;
static_assert(C == 64, "the kernels are laid out for 64 tokens");

struct ChunkParams {
  pi_ssd r;
  const float* proj;
  size_t stride;
  float* y;
  const int32_t *chunk_seqs, *chunks, *chunk0, *seq_row0, *seq_n, *seq_start, *slot;
  int dimp, vdimp, heads_cta;
  size_t row;                            // elements of a row of planes: heads * vdimp | groups * dimp (B) | groups * dimp (C)
  __nv_bfloat16 *hi, *lo;                // [chunk * C][row]
  float *dt, *F;                         // [chunk][head][C]
  float* U;                              // [chunk][head][dim][vdim]
};

struct ChunkAt {
  int seq, t0, row0, n;                  // sequence, first token of the portion, its row, tokens
};
__device__ __forceinline__ ChunkAt chunk_at(const ChunkParams& p, int c) {
  ChunkAt a;
  a.seq = p.chunk_seqs[p.chunks[2 * c]];
  a.t0 = p.chunks[2 * c + 1];
  a.row0 = p.seq_row0[a.seq] + a.t0;
  a.n = min(C, p.seq_n[a.seq] - a.t0);
  return a;
}

// Thread = one padded channel (blockIdx.x < channel blocks) or one head, over the chunk's tokens.
__global__ void __launch_bounds__(128) ssd_conv_kernel(const ChunkParams p, int channel_blocks) {
  const pi_ssd& r = p.r;
  const int chunk = blockIdx.y;
  const ChunkAt at = chunk_at(p, chunk);
  if ((int)blockIdx.x >= channel_blocks) {
    const int head = ((int)blockIdx.x - channel_blocks) * 128 + threadIdx.x;
    pi_grid_dependency_wait();
    if (head >= r.heads) return;
    if (r.decay) {
      const float a = __ldg(r.log_decay + head);
      for (int t = 0; t < C; ++t) {      // tokens past the end: no decay, no input
        p.dt[((size_t)chunk * r.heads + head) * C + t] = t < at.n ? 1.f : 0.f;
        p.F[((size_t)chunk * r.heads + head) * C + t] = a * (float)min(t + 1, at.n);
      }
      return;
    }
    const float a = -expf(__ldg(r.a_log + head)), bias = __ldg(r.dt_bias + head);
    const float* src = p.proj + (size_t)at.row0 * p.stride + r.col_dt + head;
    float* dt = p.dt + ((size_t)chunk * r.heads + head) * C;
    float* F = p.F + ((size_t)chunk * r.heads + head) * C;
    float f = 0.f;
    for (int t0 = 0; t0 < C; t0 += 8) {
      float d[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) d[j] = src[(size_t)min(t0 + j, at.n - 1) * p.stride];
#pragma unroll
      for (int j = 0; j < 8; ++j) {      // tokens past the end: no decay, no input
        const float v = t0 + j < at.n ? pi_softplus(d[j] + bias) : 0.f;
        f = fmaf(a, v, f);
        dt[t0 + j] = v;
        F[t0 + j] = f;
      }
    }
    return;
  }
  const int i = (int)blockIdx.x * 128 + threadIdx.x, inner = r.inner(), gn = r.groups * r.dim;
  int c = -1;                            // channel among x, B, C
  if (i < r.heads * p.vdimp) {
    const int h = i / p.vdimp, e = i - h * p.vdimp;
    if (e < r.vdim) c = h * r.vdim + e;
  } else if (i < (int)p.row) {
    const int k = i - r.heads * p.vdimp, g = k / p.dimp, n = k - g * p.dimp;   // g: B's groups, then C's
    if (n < r.dim) c = inner + (g < r.groups ? g * r.dim + n : gn + (g - r.groups) * r.dim + n);
  }
  const float* w = r.conv + (size_t)max(c, 0) * r.taps;   // not read without a convolution
  const float bias = c >= 0 && r.conv ? __ldg(r.conv_b + c) : 0.f;
  const int channels = r.channels();
  const bool fresh = p.seq_start[at.seq] == 0;
  const float* past = r.state + (size_t)p.slot[at.seq] * r.state_stride + r.state_off + (size_t)r.heads * r.dim * r.vdim;
  pi_grid_dependency_wait();
  if (i >= (int)p.row) return;
  const float* x = p.proj + (size_t)p.seq_row0[at.seq] * p.stride + r.col_x + max(c, 0);
  auto input = [&](int t) {              // token t of the portion
    if (t >= 0) return x[(size_t)t * p.stride];
    return fresh ? 0.f : past[(size_t)(r.taps - 1 + t) * channels + max(c, 0)];
  };
  __nv_bfloat16* hi = p.hi + (size_t)chunk * C * p.row + i;
  __nv_bfloat16* lo = p.lo + (size_t)chunk * C * p.row + i;
  auto put = [&](int t, float v) {
    v = c >= 0 && t < at.n ? v * pi_sigmoid(v) : 0.f;
    const __nv_bfloat16 h = __float2bfloat16_rn(v);
    hi[(size_t)t * p.row] = h;
    lo[(size_t)t * p.row] = __float2bfloat16_rn(v - __bfloat162float(h));
  };
  if (r.taps <= 4) {                     // the last inputs stay in registers
    float w4[4] = {0.f, 0.f, 0.f, 0.f}, u[3] = {0.f, 0.f, 0.f};
#pragma unroll
    for (int j = 0; j < 4; ++j)          // aligned to the current token: w4[3] is its own
      if (j >= 4 - r.taps) w4[j] = r.conv ? __ldg(w + j - (4 - r.taps)) : 1.f;
#pragma unroll
    for (int j = 0; j < 3; ++j)
      if (j >= 4 - r.taps) u[j] = input(at.t0 - 3 + j);
    for (int t0 = 0; t0 < C; t0 += 8) {
      float v[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = x[(size_t)(at.t0 + min(t0 + j, at.n - 1)) * p.stride];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        put(t0 + j, fmaf(w4[3], v[j], fmaf(w4[2], u[2], fmaf(w4[1], u[1], fmaf(w4[0], u[0], bias)))));
        u[0] = u[1];
        u[1] = u[2];
        u[2] = v[j];
      }
    }
  } else {
    for (int t = 0; t < C; ++t) {
      float v = bias;
      if (t < at.n)
        for (int j = 0; j < r.taps; ++j) v = fmaf(__ldg(w + j), input(at.t0 + t - r.taps + 1 + j), v);
      put(t, v);
    }
  }
}

// The same without a convolution, four channels at a time: CTA = (512 padded channels, chunk, 16 of its tokens).  Behind the
// channels: the heads' dt and F.
constexpr int kPlaneTokens = 16;
__global__ void __launch_bounds__(128) silu_planes_kernel(const ChunkParams p, int channel_blocks) {
  const pi_ssd& r = p.r;
  const int chunk = blockIdx.y, t0 = blockIdx.z * kPlaneTokens;
  const ChunkAt at = chunk_at(p, chunk);
  if ((int)blockIdx.x >= channel_blocks) {
    const int i = ((int)blockIdx.x - channel_blocks) * 128 + threadIdx.x, head = i / kPlaneTokens, t = t0 + i % kPlaneTokens;
    pi_grid_dependency_wait();
    if (head >= r.heads) return;
    p.dt[((size_t)chunk * r.heads + head) * C + t] = t < at.n ? 1.f : 0.f;   // tokens past the end: no decay, no input
    p.F[((size_t)chunk * r.heads + head) * C + t] = __ldg(r.log_decay + head) * (float)min(t + 1, at.n);
    return;
  }
  const int i = ((int)blockIdx.x * 128 + threadIdx.x) * 4, inner = r.inner(), gn = r.groups * r.dim;
  int c = -1;                            // first channel among x, B, C
  if (i < r.heads * p.vdimp) {
    const int h = i / p.vdimp, e = i - h * p.vdimp;
    if (e < r.vdim) c = h * r.vdim + e;
  } else if (i < (int)p.row) {
    const int k = i - r.heads * p.vdimp, g = k / p.dimp, n = k - g * p.dimp;   // g: B's groups, then C's
    if (n < r.dim) c = inner + (g < r.groups ? g * r.dim + n : gn + (g - r.groups) * r.dim + n);
  }
  pi_grid_dependency_wait();
  if (i >= (int)p.row) return;
  const float* x = p.proj + (size_t)at.row0 * p.stride + r.col_x + max(c, 0);
  const size_t to = (size_t)chunk * C * p.row + i;
#pragma unroll
  for (int half = 0; half < kPlaneTokens; half += 8) {
    float4 v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = *reinterpret_cast<const float4*>(x + (size_t)min(t0 + half + j, at.n - 1) * p.stride);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int t = t0 + half + j;
      const bool ok = c >= 0 && t < at.n;
      const float a[4] = {ok ? v[j].x * pi_sigmoid(v[j].x) : 0.f, ok ? v[j].y * pi_sigmoid(v[j].y) : 0.f, ok ? v[j].z * pi_sigmoid(v[j].z) : 0.f,
                          ok ? v[j].w * pi_sigmoid(v[j].w) : 0.f};
      uint2 hi, lo;
      split(a[0], a[1], hi.x, lo.x);
      split(a[2], a[3], hi.y, lo.y);
      *reinterpret_cast<uint2*>(p.hi + to + (size_t)t * p.row) = hi;
      *reinterpret_cast<uint2*>(p.lo + to + (size_t)t * p.row) = lo;
    }
  }
}

// rows x cols (a multiple of 8) of both planes into shared memory
__device__ __forceinline__ void copy_planes(const ChunkParams& p, int chunk, size_t col, int cols, __nv_bfloat16* hi, __nv_bfloat16* lo, int pitch) {
  const int pieces = cols / 8;
  const size_t from = (size_t)chunk * C * p.row + col;
  for (int i = threadIdx.x; i < C * pieces; i += kThreads) {
    const int t = i / pieces, x = (i - t * pieces) * 8;
    cp_async16(smem_addr(hi + t * pitch + x), p.hi + from + (size_t)t * p.row + x, 16);
    cp_async16(smem_addr(lo + t * pitch + x), p.lo + from + (size_t)t * p.row + x, 16);
  }
}
__device__ __forceinline__ float2 planes2(const __nv_bfloat16* hi, const __nv_bfloat16* lo) {   // two neighbours
  const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(hi)), l = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(lo));
  return make_float2(h.x + l.x, h.y + l.y);
}

__global__ void __launch_bounds__(kThreads) ssd_local_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  const pi_ssd& r = p.r;
  const int chunk = blockIdx.x, per_group = r.heads / r.groups, blocks = (per_group + p.heads_cta - 1) / p.heads_cta;
  const int group = blockIdx.y / blocks, h0 = group * per_group + (blockIdx.y % blocks) * p.heads_cta, nh = min(p.heads_cta, (group + 1) * per_group - h0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int kp = p.dimp + 8, cols = nh * p.vdimp, vp = p.heads_cta * p.vdimp + 8;
  __nv_bfloat16* khi = reinterpret_cast<__nv_bfloat16*>(smem);   // B [C][kp], x [C][vp]
  __nv_bfloat16* klo = khi + C * kp;
  __nv_bfloat16* vhi = klo + C * kp;
  __nv_bfloat16* vlo = vhi + C * vp;
  __shared__ float f[kMaxHeads][C];
  pi_grid_dependency_wait();
  copy_planes(p, chunk, (size_t)r.heads * p.vdimp + (size_t)group * p.dimp, p.dimp, khi, klo, kp);
  copy_planes(p, chunk, (size_t)h0 * p.vdimp, cols, vhi, vlo, vp);
  cp_async_commit();
  for (int i = tid; i < nh * C; i += kThreads) {
    const float* F = p.F + ((size_t)chunk * r.heads + h0) * C;
    f[i / C][i % C] = p.dt[((size_t)chunk * r.heads + h0) * C + i] * expf(F[(i / C) * C + C - 1] - F[i]);
  }
  cp_async_wait<0>();
  __syncthreads();
  for (int i = tid; i < C * cols / 2; i += kThreads) {             // x times its weight at the chunk's end
    const int t = i / (cols / 2), e = (i - t * (cols / 2)) * 2, at = t * vp + e;
    const float w = f[e / p.vdimp][t];
    const float2 v = planes2(vhi + at, vlo + at);
    split(v.x * w, v.y * w, *reinterpret_cast<uint32_t*>(vhi + at), *reinterpret_cast<uint32_t*>(vlo + at));
  }
  __syncthreads();
  const int mt = p.dimp / 16, nt = cols / 16;
  for (int item = warp; item < mt * nt; item += kWarps) {
    const int m0 = (item / nt) * 16, n0 = (item % nt) * 16;
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int k = 0; k < C; k += 16) {
      uint32_t ah[4], al[4], bh[4], bo[4];
      const int ar = k + (lane & 7) + (lane >> 4) * 8, ac = m0 + ((lane >> 3) & 1) * 8;   // B^T, stored token-major
      ldsm4_t(ah, smem_addr(khi + ar * kp + ac));
      ldsm4_t(al, smem_addr(klo + ar * kp + ac));
      const int br = k + (lane & 7) + ((lane >> 3) & 1) * 8, bc = n0 + (lane >> 4) * 8;
      ldsm4_t(bh, smem_addr(vhi + br * vp + bc));
      ldsm4_t(bo, smem_addr(vlo + br * vp + bc));
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        mma(acc[j], ah[0], ah[1], ah[2], ah[3], bh[2 * j], bh[2 * j + 1]);
        mma(acc[j], al[0], al[1], al[2], al[3], bh[2 * j], bh[2 * j + 1]);
        mma(acc[j], ah[0], ah[1], ah[2], ah[3], bo[2 * j], bo[2 * j + 1]);
      }
    }
    const int h = n0 / p.vdimp, e0 = n0 - h * p.vdimp;
    float* U = p.U + ((size_t)chunk * r.heads + h0 + h) * r.dim * r.vdim;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int n = m0 + (lane >> 2) + i * 8, e = e0 + j * 8 + (lane & 3) * 2;
        if (n >= r.dim) continue;
        if (r.vdim % 2 == 0) {
          if (e < r.vdim) *reinterpret_cast<float2*>(U + (size_t)n * r.vdim + e) = make_float2(acc[j][2 * i], acc[j][2 * i + 1]);
        } else {
          if (e < r.vdim) U[(size_t)n * r.vdim + e] = acc[j][2 * i];
          if (e + 1 < r.vdim) U[(size_t)n * r.vdim + e + 1] = acc[j][2 * i + 1];
        }
      }
  }
}

__device__ __forceinline__ uint32_t pack_planes(float v) {   // hi in the lower half, lo in the upper
  const __nv_bfloat16 h = __float2bfloat16_rn(v), l = __float2bfloat16_rn(v - __bfloat162float(h));
  return (uint32_t)__bfloat16_as_ushort(h) | ((uint32_t)__bfloat16_as_ushort(l) << 16);
}

// Thread = V consecutive state elements of one head.
template <int V>
__global__ void __launch_bounds__(256) ssd_pass_kernel(const ChunkParams p) {
  const pi_ssd& r = p.r;
  const int cs = blockIdx.z, head = blockIdx.y, seq = p.chunk_seqs[cs], per_head = r.dim * r.vdim, i = (blockIdx.x * 256 + threadIdx.x) * V;
  const int c0 = p.chunk0[cs], c1 = p.chunk0[cs + 1];
  const bool live = i < per_head;
  float* S = r.state + (size_t)p.slot[seq] * r.state_stride + r.state_off + (size_t)head * per_head + i;
  float s[V];
#pragma unroll
  for (int j = 0; j < V; ++j) s[j] = 0.f;
  if (live && p.seq_start[seq] != 0) {
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] = S[j];
  }
  pi_grid_dependency_wait();
  if (!live) return;
  constexpr int A = 8;                   // chunks fetched ahead
  for (int c = c0; c < c1; c += A) {
    float u[A][V], keep[A];
#pragma unroll
    for (int k = 0; k < A; ++k) {
      const size_t ch = (size_t)min(c + k, c1 - 1) * r.heads + head;
      const float* src = p.U + ch * per_head + i;
      if (V == 4) {
        const float4 v = *reinterpret_cast<const float4*>(src);
        u[k][0] = v.x;
        u[k][1 % V] = v.y;
        u[k][2 % V] = v.z;
        u[k][3 % V] = v.w;
      } else {
        u[k][0] = src[0];
      }
      keep[k] = p.F[ch * C + C - 1];
    }
#pragma unroll
    for (int k = 0; k < A; ++k) {
      if (c + k >= c1) break;
      uint32_t* dst = reinterpret_cast<uint32_t*>(p.U + ((size_t)(c + k) * r.heads + head) * per_head + i);
      if (V == 4) *reinterpret_cast<uint4*>(dst) = make_uint4(pack_planes(s[0]), pack_planes(s[1 % V]), pack_planes(s[2 % V]), pack_planes(s[3 % V]));
      else dst[0] = pack_planes(s[0]);
      const float f = expf(keep[k]);
#pragma unroll
      for (int j = 0; j < V; ++j) s[j] = fmaf(f, s[j], u[k][j]);
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) S[j] = s[j];
}

__global__ void __launch_bounds__(kThreads, 2) ssd_output_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  const pi_ssd& r = p.r;
  const int chunk = blockIdx.x, per_group = r.heads / r.groups, blocks = (per_group + p.heads_cta - 1) / p.heads_cta;
  const int group = blockIdx.y / blocks, h0 = group * per_group + (blockIdx.y % blocks) * p.heads_cta, nh = min(p.heads_cta, (group + 1) * per_group - h0);
  const ChunkAt at = chunk_at(p, chunk);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int kp = p.dimp + 8, vp = kVS + 8, nks = p.dimp / 16;
  __nv_bfloat16* chi = reinterpret_cast<__nv_bfloat16*>(smem);       // C [C][kp]
  __nv_bfloat16* clo = chi + C * kp;
  __nv_bfloat16* bhi = clo + C * kp;                                 // B [C][kp]; later, in its place, the state [dimp][vp]
  __nv_bfloat16* blo = bhi + C * kp;
  __nv_bfloat16* shi = bhi;
  __nv_bfloat16* slo = shi + p.dimp * vp;
  __nv_bfloat16* xhi = bhi + 2 * max(C * kp, p.dimp * vp);           // x [C][vp]
  __nv_bfloat16* xlo = xhi + C * vp;
  float* A = reinterpret_cast<float*>(xlo + C * vp);                 // C . B [C][kApitch]
  __shared__ float sF[C], sdt[C];
  pi_grid_dependency_wait();
  const size_t col_b = (size_t)r.heads * p.vdimp + (size_t)group * p.dimp;
  copy_planes(p, chunk, col_b + (size_t)r.groups * p.dimp, p.dimp, chi, clo, kp);
  copy_planes(p, chunk, col_b, p.dimp, bhi, blo, kp);
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  for (int item = warp; item < 10; item += kWarps) {                 // 16 x 16 tokens at a time, on and below the diagonal
    int I = 0, J = item;
    while (J > I) J -= ++I;
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 2
    for (int k = 0; k < nks; ++k) {
      uint32_t ah[4], al[4], bh[4], bo[4];
      const int ar = (I * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kp + k * 16 + (lane >> 4) * 8;
      ldsm4(ah, smem_addr(chi + ar));
      ldsm4(al, smem_addr(clo + ar));
      const int br = (J * 16 + (lane & 7) + ((lane >> 4) << 3)) * kp + k * 16 + ((lane >> 3) & 1) * 8;
      ldsm4(bh, smem_addr(bhi + br));
      ldsm4(bo, smem_addr(blo + br));
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        mma(acc[j], ah[0], ah[1], ah[2], ah[3], bh[2 * j], bh[2 * j + 1]);
        mma(acc[j], al[0], al[1], al[2], al[3], bh[2 * j], bh[2 * j + 1]);
        mma(acc[j], ah[0], ah[1], ah[2], ah[3], bo[2 * j], bo[2 * j + 1]);
      }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 2; ++i)
        *reinterpret_cast<float2*>(A + (I * 16 + (lane >> 2) + 8 * i) * kApitch + J * 16 + j * 8 + (lane & 3) * 2) = make_float2(acc[j][2 * i], acc[j][2 * i + 1]);
  }

  // warp = (16 tokens, half of the 64 value columns of a pass)
  const int I = warp >> 1, half = warp & 1, rt = I * 16 + (lane >> 2);
  for (int h = h0; h < h0 + nh; ++h) {
    const size_t ch = (size_t)chunk * r.heads + h;
    const float skip = r.d ? __ldg(r.d + h) : 0.f;
    for (int c0 = 0; c0 < r.vdim; c0 += kVS) {
      const int cols = min(kVS, p.vdimp - c0);
      __syncthreads();                   // the last pass (or the scores) has read what is overwritten now
      copy_planes(p, chunk, (size_t)h * p.vdimp + c0, cols, xhi, xlo, vp);
      cp_async_commit();
      if (c0 == 0 && tid < C) {
        sF[tid] = p.F[ch * C + tid];
        sdt[tid] = p.dt[ch * C + tid];
      }
      const uint32_t* U = reinterpret_cast<const uint32_t*>(p.U) + ch * r.dim * r.vdim + c0;
      if (r.vdim % 4 == 0) {
        const int c4 = cols / 4, count = p.dimp * c4;
        constexpr int B = 4;
        for (int i0 = tid; i0 < count; i0 += B * kThreads) {
          uint4 v[B];
#pragma unroll
          for (int b = 0; b < B; ++b) {  // outside reads the first element and counts as zero
            const int i = min(i0 + b * kThreads, count - 1), n = i / c4, e = (i - n * c4) * 4;
            const bool ok = n < r.dim && c0 + e < r.vdim;
            v[b] = *reinterpret_cast<const uint4*>(ok ? U + (size_t)n * r.vdim + e : U);
            if (!ok) v[b] = make_uint4(0, 0, 0, 0);
          }
#pragma unroll
          for (int b = 0; b < B; ++b) {
            const int i = i0 + b * kThreads, n = i / c4, e = (i - n * c4) * 4;
            if (i >= count) break;
            *reinterpret_cast<uint2*>(shi + n * vp + e) = make_uint2(__byte_perm(v[b].x, v[b].y, 0x5410), __byte_perm(v[b].z, v[b].w, 0x5410));
            *reinterpret_cast<uint2*>(slo + n * vp + e) = make_uint2(__byte_perm(v[b].x, v[b].y, 0x7632), __byte_perm(v[b].z, v[b].w, 0x7632));
          }
        }
      } else {
        for (int i = tid; i < p.dimp * cols; i += kThreads) {
          const int n = i / cols, e = i - n * cols;
          const uint32_t v = n < r.dim && c0 + e < r.vdim ? U[(size_t)n * r.vdim + e] : 0u;
          shi[n * vp + e] = __ushort_as_bfloat16((unsigned short)(v & 0xffffu));
          slo[n * vp + e] = __ushort_as_bfloat16((unsigned short)(v >> 16));
        }
      }
      cp_async_wait<0>();
      __syncthreads();
      if (half * 32 >= cols) continue;   // uniform for the warp; every barrier above is met by all
      float acc[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
      auto products = [&](const uint32_t* ah, const uint32_t* al, const __nv_bfloat16* hi, const __nv_bfloat16* lo, int k0) {
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          if (half * 32 + j * 8 >= cols) break;
          uint32_t bh[4], bo[4];
          const int b = (k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * vp + half * 32 + j * 8 + (lane >> 4) * 8;
          ldsm4_t(bh, smem_addr(hi + b));
          ldsm4_t(bo, smem_addr(lo + b));
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            mma(acc[j + x], ah[0], ah[1], ah[2], ah[3], bh[2 * x], bh[2 * x + 1]);
            mma(acc[j + x], al[0], al[1], al[2], al[3], bh[2 * x], bh[2 * x + 1]);
            mma(acc[j + x], ah[0], ah[1], ah[2], ah[3], bo[2 * x], bo[2 * x + 1]);
          }
        }
      };
#pragma unroll 2
      for (int k = 0; k < nks; ++k) {
        uint32_t ah[4], al[4];
        const int ar = (I * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kp + k * 16 + (lane >> 4) * 8;
        ldsm4(ah, smem_addr(chi + ar));
        ldsm4(al, smem_addr(clo + ar));
        products(ah, al, shi, slo, k * 16);
      }
      const float F0 = sF[rt], F1 = sF[rt + 8], g0 = expf(F0), g1 = expf(F1);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[j][0] *= g0;
        acc[j][1] *= g0;
        acc[j][2] *= g1;
        acc[j][3] *= g1;
      }
#pragma unroll 1
      for (int J = 0; J <= I; ++J) {
        uint32_t ah[4], al[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {    // a0: row, a1: row + 8, a2 / a3: tokens + 8
          const int t = rt + (q & 1) * 8, s = J * 16 + (lane & 3) * 2 + (q >> 1) * 8;
          const float Ft = q & 1 ? F1 : F0;
          const float2 a = *reinterpret_cast<const float2*>(A + t * kApitch + s);
          const float w0 = s <= t ? a.x * expf(Ft - sF[s]) * sdt[s] : 0.f, w1 = s + 1 <= t ? a.y * expf(Ft - sF[s + 1]) * sdt[s + 1] : 0.f;
          split(w0, w1, ah[q], al[q]);
        }
        products(ah, al, xhi, xlo, J * 16);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = rt + 8 * i;
        if (t >= at.n) continue;
        const float* z = p.proj + (size_t)(at.row0 + t) * p.stride + r.col_z + (size_t)h * r.vdim;
        float* y = p.y + (size_t)(at.row0 + t) * r.inner() + (size_t)h * r.vdim;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int e = half * 32 + j * 8 + (lane & 3) * 2;
          if (e >= cols) break;
          const float2 x = planes2(xhi + t * vp + e, xlo + t * vp + e);
#pragma unroll
          for (int k = 0; k < 2; ++k) {
            if (c0 + e + k >= r.vdim) break;
            float v = fmaf(skip, k ? x.y : x.x, acc[j][2 * i + k]);
            if (!r.gate_last) {
              const float g = z[c0 + e + k];
              v *= g * pi_sigmoid(g);
            }
            y[c0 + e + k] = v;
          }
        }
      }
    }
  }
}

size_t local_smem(const ChunkParams& p) { return (size_t)4 * C * (p.dimp + 8 + p.heads_cta * p.vdimp + 8); }
size_t output_smem(const ChunkParams& p) {
  const int vp = kVS + 8;
  return (size_t)4 * C * (p.dimp + 8) + (size_t)4 * std::max(C * (p.dimp + 8), p.dimp * vp) + (size_t)4 * C * vp + (size_t)4 * C * kApitch;
}
void sizes(ChunkParams& p) {
  p.dimp = (p.r.dim + 15) / 16 * 16;
  p.vdimp = (p.r.vdim + 15) / 16 * 16;
  p.row = (size_t)p.r.heads * p.vdimp + 2 * (size_t)p.r.groups * p.dimp;
  p.heads_cta = std::min(kMaxHeads, p.r.heads / p.r.groups);
  while (p.heads_cta > 1 && local_smem(p) > 110 * 1024) --p.heads_cta;
}
cudaError_t grant(pi_ctx* ctx, void (*k)(const ChunkParams), size_t smem, pi_smem_grant& g) {
  if (smem <= g.of(ctx) || smem <= kSmemFree) return cudaSuccess;
  g.of(ctx) = smem;
  return cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

}  // namespace

bool pi_ssd_chunked(const pi_ctx* ctx, const pi_ssd& r, int compute) {
  ChunkParams p = {};
  p.r = r;
  sizes(p);
  return compute == PI_BF16 && r.dim <= kMaxDim && std::max(local_smem(p), output_smem(p)) + 4096 <= ctx->smem_optin;
}

size_t pi_ssd_scratch_floats(const pi_ssd& r, int n_chunks) {
  if (!n_chunks) return 0;
  ChunkParams p = {};
  p.r = r;
  sizes(p);
  return (size_t)n_chunks * (C * p.row + 2 * (size_t)r.heads * C + (size_t)r.heads * r.dim * r.vdim) + 64;
}

pi_status pi_launch_ssd_chunks(pi_ctx* ctx, const pi_ssd& r, const float* proj, size_t stride, float* y, const pi_seq_batch& b, float* scratch) {
  static pi_smem_grant g1, g2;
  PI_REQUIRE(ctx, scratch, "long portions need scratch");
  ChunkParams p = {};
  p.r = r;
  sizes(p);
  p.proj = proj;
  p.stride = stride;
  p.y = y;
  p.chunk_seqs = b.chunk_seqs;
  p.chunks = b.chunks;
  p.chunk0 = b.chunk0;
  p.seq_row0 = b.seq_row0;
  p.seq_n = b.seq_n;
  p.seq_start = b.seq_start;
  p.slot = b.slot;
  const size_t planes = (size_t)b.n_chunks * C * p.row, gates = (size_t)b.n_chunks * r.heads * C;   // multiples of 4
  p.hi = reinterpret_cast<__nv_bfloat16*>(scratch);
  p.lo = p.hi + planes;
  p.dt = scratch + planes;
  p.F = p.dt + gates;
  p.U = p.F + gates;
  const int channel_blocks = (int)((p.row + 127) / 128), head_blocks = (r.heads + 127) / 128;
  if (!r.conv && r.decay && r.vdim % 4 == 0 && r.dim % 4 == 0 && r.col_x % 4 == 0 && stride % 4 == 0) {
    const int four = (int)((p.row + 511) / 512), heads = (r.heads * kPlaneTokens + 127) / 128;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, silu_planes_kernel, dim3(four + heads, b.n_chunks, C / kPlaneTokens), dim3(128), 0, 1, p, four));
  } else {
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, ssd_conv_kernel, dim3(channel_blocks + head_blocks, b.n_chunks), dim3(128), 0, 1, p, channel_blocks));
  }
  const int per_group = r.heads / r.groups, blocks = r.groups * ((per_group + p.heads_cta - 1) / p.heads_cta), per_head = r.dim * r.vdim;
  const size_t s1 = local_smem(p), s2 = output_smem(p);
  PI_CUDA(ctx, grant(ctx, ssd_local_kernel, s1, g1));
  PI_CUDA(ctx, grant(ctx, ssd_output_kernel, s2, g2));
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, ssd_local_kernel, dim3(b.n_chunks, blocks), dim3(kThreads), s1, 1, p));
  const bool vec = per_head % 4 == 0;
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, vec ? ssd_pass_kernel<4> : ssd_pass_kernel<1>, dim3((per_head / (vec ? 4 : 1) + 255) / 256, r.heads, b.n_chunk_seqs), dim3(256), 0,
                                  1, p));
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, ssd_output_kernel, dim3(b.n_chunks, blocks), dim3(kThreads), s2, 1, p));
  return PI_OK;
}
