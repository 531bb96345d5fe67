// Portions of many tokens through the recurrences of pi_recurrent.cu, in chunks of 64 tokens that run side by side:
//
//   1. recur_local_kernel    per chunk and head: what the chunk adds to the state, U = K~^T V (K~: keys decayed to the
//                            chunk's end), and the decay of the chunk as a whole
//   2. recur_pass_kernel     per state element: the state in front of every chunk, one pass over the chunks; U is
//                            overwritten with it, the final state goes to the slot
//   3. recur_output_kernel   per chunk and head: O = Q~ S + (causal part inside the chunk) V, normaliser, head norm, gate
//
// The recurrence is f32: every operand of a tensor-core product (mma.sync) is a pair of bf16 planes, hi + lo (16 bits),
// three products each.  All exponents are differences that are never positive, whatever the gates:
//   GLA    b = running sum of the log decays inside a 16-token subchunk, tot = its end.  A key is kept decayed to the end of
//          its subchunk, k e^(tot_J - b_s), a query decayed from the start of its own, q e^(b_t); what lies between the two is
//          a factor per channel, E_IJ = exp(sum of tot over the subchunks between).  Inside one subchunk E = e^(-tot), which
//          is safe while tot > -60; a subchunk that decays further is summed pair by pair.
//   mLSTM  F = running sum of the log forget gates, G_t = max over s <= t of F_t - F_s + i_s; then m_t = max(F_t + m, G_t) with
//          m in front of the chunk, and the weight of key s at token t is exp(F_t - F_s + i_s - m_t).
#include <math.h>

#include <algorithm>

#include "pi_layered.cuh"
#include "pi_mma.cuh"

namespace {
using namespace pi_mma;

constexpr int C = kRecurrenceChunk, SUB = 16, NSUB = C / SUB;
constexpr int kChunkThreads = 256, kChunkWarps = 8;
constexpr int kVS = 64;               // value columns per pass of the output kernel
constexpr int kMaxDim = 128, kMaxVdim = 256;
constexpr float kSafeDecay = -60.f;
constexpr int kFactors = NSUB * (NSUB + 1) / 2 + NSUB;
static_assert(C == 64, "the kernels are laid out for 64 tokens");

struct ChunkParams {
  pi_recurrence r;
  const float* proj;
  size_t stride;
  __nv_bfloat16* out;
  size_t out_stride;
  const int32_t *chunk_seqs, *chunks, *chunk0, *seq_row0, *seq_n, *seq_start, *slot;
  // scratch, per chunk and head
  float* U;        // [chunk][head][dim][vdim]
  float* nU;       // [chunk][head][dim]            mLSTM
  float* decay;    // [chunk][head][dim]            GLA: of the whole chunk
  float* FG;       // [chunk][head][2]              mLSTM: F and G at the chunk's end
  float* m_in;     // [chunk][head]                 mLSTM
  int dimp, vdimp;   // rounded up to 16
  bool vec_k, vec_v;   // 16-byte loads of keys and queries / of values, output gates and state rows
};

struct ChunkAt {
  int seq, row0, n;   // sequence, first row, tokens
};
__device__ __forceinline__ ChunkAt chunk_at(const ChunkParams& p, int c) {
  ChunkAt a;
  a.seq = p.chunk_seqs[p.chunks[2 * c]];
  const int t0 = p.chunks[2 * c + 1];
  a.row0 = p.seq_row0[a.seq] + t0;
  a.n = min(C, p.seq_n[a.seq] - t0);
  return a;
}

// GLA: bl[t][d] = running sum of the log decays inside t's subchunk (inclusive), tot[J][d] its end.  Tokens past the
// chunk's end do not decay.
__device__ __forceinline__ void gla_decays(const ChunkParams& p, const ChunkAt& at, int head, float* low, float* bl, float* tot) {
  const pi_recurrence& r = p.r;
  for (int i = threadIdx.x; i < C * r.rank; i += kChunkThreads) {
    const int t = i / r.rank, j = i - t * r.rank;
    low[i] = t < at.n ? __ldg(p.proj + (size_t)(at.row0 + t) * p.stride + r.col_low + j) : 0.f;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < NSUB * p.dimp; i += kChunkThreads) {
    const int J = i / p.dimp, d = i - J * p.dimp, c = head * r.dim + d;
    float z[SUB];
#pragma unroll
    for (int t = 0; t < SUB; ++t) z[t] = 0.f;
    if (d < r.dim) {
      const float* w = r.a2 + (size_t)c * r.rank;
      for (int j = 0; j < r.rank; ++j) {
        const float wj = __ldg(w + j);
#pragma unroll
        for (int t = 0; t < SUB; ++t) z[t] = fmaf(wj, low[(J * SUB + t) * r.rank + j], z[t]);
      }
      const float bias = __ldg(r.a2_b + c);
#pragma unroll
      for (int t = 0; t < SUB; ++t) z[t] = J * SUB + t < at.n ? pi_log_sigmoid(z[t] + bias) / r.tau : 0.f;
    }
    float b = 0.f;
#pragma unroll
    for (int t = 0; t < SUB; ++t) {
      b += z[t];
      bl[(J * SUB + t) * p.dimp + d] = b;
    }
    tot[J * p.dimp + d] = b;
  }
  __syncthreads();
}

// mLSTM: li[t], F[t], G[t] of the chunk (first warp; every lane holds two tokens).
__device__ __forceinline__ void mlstm_gates(const ChunkParams& p, const ChunkAt& at, int head, float* li, float* F, float* G) {
  const pi_recurrence& r = p.r;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    float f[2], g[2], iv[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int t = 2 * lane + j;
      f[j] = 0.f;
      g[j] = iv[j] = -INFINITY;       // tokens past the end: no decay, no input
      if (t < at.n) {
        const float* x = p.proj + (size_t)(at.row0 + t) * p.stride;
        iv[j] = r.gate_cap * tanhf((x[r.col_i + head] + r.i_b[head]) / r.gate_cap);
        f[j] = pi_log_sigmoid(r.gate_cap * tanhf((x[r.col_f + head] + r.f_b[head]) / r.gate_cap));
        g[j] = iv[j];
      }
    }
    float sf = f[0] + f[1], sg = fmaxf(f[1] + g[0], g[1]);     // the lane's two tokens as one step
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pf = __shfl_up_sync(0xffffffffu, sf, o), pg = __shfl_up_sync(0xffffffffu, sg, o);
      if (lane >= o) {
        sg = fmaxf(sf + pg, sg);
        sf += pf;
      }
    }
    float ef = __shfl_up_sync(0xffffffffu, sf, 1), eg = __shfl_up_sync(0xffffffffu, sg, 1);   // in front of the lane's tokens
    if (lane == 0) {
      ef = 0.f;
      eg = -INFINITY;
    }
    li[2 * lane] = iv[0];
    li[2 * lane + 1] = iv[1];
    F[2 * lane] = ef + f[0];
    F[2 * lane + 1] = sf;
    G[2 * lane] = fmaxf(f[0] + eg, g[0]);
    G[2 * lane + 1] = sg;
  }
  __syncthreads();
}

__device__ __forceinline__ void store_split(__nv_bfloat16* hi, __nv_bfloat16* lo, int i, float v) {
  const __nv_bfloat16 h = __float2bfloat16_rn(v);
  hi[i] = h;
  lo[i] = __float2bfloat16_rn(v - __bfloat162float(h));
}
__device__ __forceinline__ void store_split4(__nv_bfloat16* hi, __nv_bfloat16* lo, int i, float4 v) {   // i: a multiple of 4
  uint2 h, l;
  split(v.x, v.y, h.x, l.x);
  split(v.z, v.w, h.y, l.y);
  *reinterpret_cast<uint2*>(hi + i) = h;
  *reinterpret_cast<uint2*>(lo + i) = l;
}

// A [rows][cols] piece of a matrix (cols a multiple of 4, zero outside the first `have_rows` rows and `have_cols` columns),
// walked by the CTA four columns at a time: use(row, col, float4).  With `vec` (16-byte loads possible, have_cols a multiple
// of 4) several loads are in flight per thread before the first of them is used; instead of branching, what is outside reads
// `safe`, any valid 16-byte aligned address.
template <typename F>
__device__ __forceinline__ void staged(const float* safe, const float* src, size_t ld, int rows, int cols, int have_rows, int have_cols, bool vec, F&& use) {
  constexpr int U = 4;
  const int c4 = cols >> 2, count = rows * c4;
  if (vec) {
    for (int i0 = threadIdx.x; i0 < count; i0 += U * kChunkThreads) {
      float4 v[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = min(i0 + u * kChunkThreads, count - 1), r = i / c4, c = (i - r * c4) * 4;
        const bool ok = r < have_rows && c < have_cols;
        v[u] = __ldg(reinterpret_cast<const float4*>(ok ? src + (size_t)r * ld + c : safe));
        if (!ok) v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = i0 + u * kChunkThreads, r = i / c4;
        if (i < count) use(r, (i - r * c4) * 4, v[u]);
      }
    }
  } else {
    for (int i = threadIdx.x; i < count; i += kChunkThreads) {
      const int r = i / c4, c = (i - r * c4) * 4;
      float x[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) x[j] = (r < have_rows && c + j < have_cols) ? __ldg(src + (size_t)r * ld + c + j) : 0.f;
      use(r, c, make_float4(x[0], x[1], x[2], x[3]));
    }
  }
}

// value columns [c0, c0 + cols) of the chunk as two planes [C][pitch]
__device__ __forceinline__ void load_v(const ChunkParams& p, const ChunkAt& at, int head, int c0, int cols, __nv_bfloat16* hi, __nv_bfloat16* lo,
                                       int pitch) {
  const float* src = p.proj + (size_t)at.row0 * p.stride + p.r.col_v + (size_t)head * p.r.vdim + c0;
  staged(p.proj, src, p.stride, C, cols, at.n, p.r.vdim - c0, p.vec_v, [&](int t, int e, float4 v) { store_split4(hi, lo, t * pitch + e, v); });
}

template <int KIND>
__global__ void __launch_bounds__(kChunkThreads) recur_local_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const pi_recurrence& r = p.r;
  const int head = blockIdx.y, chunk = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const ChunkAt at = chunk_at(p, chunk);
  const int kp = p.dimp + 8, vp = p.vdimp + 8;
  __nv_bfloat16* khi = reinterpret_cast<__nv_bfloat16*>(smem_raw);   // K~ planes [C][kp], V planes [C][vp]
  __nv_bfloat16* klo = khi + C * kp;
  __nv_bfloat16* vhi = klo + C * kp;
  __nv_bfloat16* vlo = vhi + C * vp;
  float* bl = reinterpret_cast<float*>(vlo + C * vp);                // GLA: [C][dimp], [NSUB][dimp], [C][rank]
  float* tot = bl + C * p.dimp;
  float* low = tot + NSUB * p.dimp;
  __shared__ float li[C], F[C], G[C];
  pi_grid_dependency_wait();
  const size_t ch = (size_t)chunk * r.heads + head;
  if (KIND == PI_REC_GLA) {
    gla_decays(p, at, head, low, bl, tot);
    for (int d = tid; d < r.dim; d += kChunkThreads) {
      float s = 0.f;
      for (int J = 0; J < NSUB; ++J) s += tot[J * p.dimp + d];
      p.decay[ch * r.dim + d] = expf(s);
    }
  } else {
    mlstm_gates(p, at, head, li, F, G);
    if (tid == 0) {
      p.FG[2 * ch] = F[C - 1];
      p.FG[2 * ch + 1] = G[C - 1];
    }
  }
  const float* ksrc = p.proj + (size_t)at.row0 * p.stride + r.col_k + (size_t)head * r.dim;
  staged(p.proj, ksrc, p.stride, C, p.dimp, at.n, r.dim, p.vec_k,
         [&](int t, int d, float4 v) {
           if (KIND == PI_REC_GLA) {
             float4 e = make_float4(0.f, 0.f, 0.f, 0.f);
             for (int J = t / SUB; J < NSUB; ++J) {
               const float4 x = *reinterpret_cast<const float4*>(tot + J * p.dimp + d);
               e = make_float4(e.x + x.x, e.y + x.y, e.z + x.z, e.w + x.w);
             }
             const float4 b = *reinterpret_cast<const float4*>(bl + t * p.dimp + d);
             v = make_float4(v.x * expf(e.x - b.x), v.y * expf(e.y - b.y), v.z * expf(e.z - b.z), v.w * expf(e.w - b.w));
           } else {
             const float f = t < at.n ? expf(F[C - 1] - F[t] + li[t] - G[C - 1]) : 0.f;   // the chunk's state is kept times e^-G
             v = make_float4(v.x * f, v.y * f, v.z * f, v.w * f);
           }
           store_split4(khi, klo, t * kp + d, v);
         });
  load_v(p, at, head, 0, p.vdimp, vhi, vlo, vp);
  __syncthreads();
  if (KIND == PI_REC_MLSTM) {
    for (int d = tid; d < r.dim; d += kChunkThreads) {
      float s = 0.f;
      for (int t = 0; t < C; ++t) s += __bfloat162float(khi[t * kp + d]) + __bfloat162float(klo[t * kp + d]);
      p.nU[ch * r.dim + d] = s;
    }
  }
  // U: 16 channels x 16 value columns at a time
  float* U = p.U + ch * r.dim * r.vdim;
  const int mt = p.dimp / 16, nt = p.vdimp / 16;
  for (int item = warp; item < mt * nt; item += kChunkWarps) {
    const int m0 = (item / nt) * 16, n0 = (item % nt) * 16;
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int k = 0; k < C; k += 16) {
      uint32_t ah[4], al[4], bh[4], bo[4];
      // K~^T: tiles (channels 0-7, tokens 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15), stored token-major
      const int ar = k + (lane & 7) + (lane >> 4) * 8, ac = m0 + ((lane >> 3) & 1) * 8;
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
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = m0 + (lane >> 2) + (i >> 1) * 8, e = n0 + j * 8 + (lane & 3) * 2 + (i & 1);
        if (d < r.dim && e < r.vdim) U[(size_t)d * r.vdim + e] = acc[j][i];
      }
  }
}

// Thread = V consecutive state elements of one head (blockIdx.x < elem_blocks), or one channel of n (the blocks behind
// them; channel 0 also notes m in front of every chunk).
template <int KIND, int V>
__global__ void __launch_bounds__(256) recur_pass_kernel(const ChunkParams p, int elem_blocks) {
  const pi_recurrence& r = p.r;
  const int cs = blockIdx.z, head = blockIdx.y, seq = p.chunk_seqs[cs];
  const int c0 = p.chunk0[cs], c1 = p.chunk0[cs + 1];
  const bool fresh = p.seq_start[seq] == 0, is_n = (int)blockIdx.x >= elem_blocks;
  const int per_head = r.dim * r.vdim;
  const int i = is_n ? ((int)blockIdx.x - elem_blocks) * 256 + threadIdx.x : (blockIdx.x * 256 + threadIdx.x) * V;
  float* st = r.state + (size_t)p.slot[seq] * r.state_stride + r.state_off;
  float* S = st + (size_t)head * per_head;
  float* nst = st + (size_t)r.heads * per_head + (size_t)head * r.dim;
  float* mst = st + (size_t)r.heads * per_head + (size_t)r.heads * r.dim + head;
  const bool live = i < (is_n ? r.dim : per_head);
  float s[V];
#pragma unroll
  for (int j = 0; j < V; ++j) s[j] = 0.f;
  float m = 0.f;
  if (live && !fresh) {
    if (is_n) {
      s[0] = nst[i];
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) s[j] = S[i + j];
    }
  }
  if (KIND == PI_REC_MLSTM && !fresh) m = *mst;
  pi_grid_dependency_wait();
  if (!live) return;
  const int d = is_n ? i : i / r.vdim;      // V divides vdim
  constexpr int A = 4;                      // chunks fetched ahead
  float u[A][V], k1[A], k2[A];
  auto at = [&](int c) { return is_n ? p.nU + ((size_t)c * r.heads + head) * r.dim + i : p.U + ((size_t)c * r.heads + head) * per_head + i; };
  auto fetch = [&](int c, int slot) {
    const float* src = at(c);
    if (V == 4 && !is_n) {
      const float4 v = *reinterpret_cast<const float4*>(src);
      u[slot][0] = v.x;
      if (V > 1) {
        u[slot][1 % V] = v.y;
        u[slot][2 % V] = v.z;
        u[slot][3 % V] = v.w;
      }
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) u[slot][j] = (j == 0 || !is_n) ? src[j] : 0.f;
    }
    const size_t ch = (size_t)c * r.heads + head;
    if (KIND == PI_REC_GLA) {
      k1[slot] = p.decay[ch * r.dim + d];
    } else {
      k1[slot] = p.FG[2 * ch];
      k2[slot] = p.FG[2 * ch + 1];
    }
  };
  for (int c = c0; c < c1; c += A) {
#pragma unroll
    for (int j = 0; j < A; ++j)
      if (c + j < c1) fetch(c + j, j);
#pragma unroll
    for (int j = 0; j < A; ++j) {
      if (c + j >= c1) break;
      float* dst = const_cast<float*>(at(c + j));
      if (V == 4 && !is_n) {
        *reinterpret_cast<float4*>(dst) = make_float4(s[0], s[1 % V], s[2 % V], s[3 % V]);
      } else {
#pragma unroll
        for (int x = 0; x < V; ++x)
          if (x == 0 || !is_n) dst[x] = s[x];
      }
      float keep = k1[j], put = 1.f;
      if (KIND == PI_REC_MLSTM) {
        if (is_n && i == 0) p.m_in[(size_t)(c + j) * r.heads + head] = m;
        const float mn = fmaxf(k1[j] + m, k2[j]);
        keep = expf(k1[j] + m - mn);
        put = expf(k2[j] - mn);
        m = mn;
      }
#pragma unroll
      for (int x = 0; x < V; ++x) s[x] = fmaf(keep, s[x], put * u[j][x]);
    }
  }
  if (is_n) {
    nst[i] = s[0];   // m is stored by the output kernel: here other blocks may still be reading it
  } else {
#pragma unroll
    for (int j = 0; j < V; ++j) S[i + j] = s[j];
  }
}

// NS: passes of 64 value columns.  (Loops are kept rolled where they can be: the kernel is otherwise bound by instruction
// fetch.)
template <int KIND, int NS>
__global__ void __launch_bounds__(kChunkThreads) recur_output_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const pi_recurrence& r = p.r;
  const int head = blockIdx.y, chunk = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const ChunkAt at = chunk_at(p, chunk);
  const size_t ch = (size_t)chunk * r.heads + head;
  const int qp = p.dimp + 4, kp = p.dimp + 8, ap = C + 8, vp = kVS + 8, nks = p.dimp / 16;
  float* qf = reinterpret_cast<float*>(smem_raw);                   // [C][qp] queries (GLA: decayed from their subchunk's start)
  float* tot = qf + C * qp;                                         // GLA: [NSUB][dimp], then the factors [kFactors][dimp]
  float* fac = tot + NSUB * p.dimp;
  __nv_bfloat16* khi = reinterpret_cast<__nv_bfloat16*>(fac + (KIND == PI_REC_GLA ? kFactors * p.dimp : 0));   // [C][kp] x 2, later
  __nv_bfloat16* klo = khi + C * kp;                                //   in its place: the state [dimp][vp] x 2
  __nv_bfloat16* shi = khi;
  __nv_bfloat16* slo = shi + p.dimp * vp;
  __nv_bfloat16* ahi = khi + 2 * max(C * kp, p.dimp * vp);          // [C][ap] x 2: weights inside the chunk
  __nv_bfloat16* alo = ahi + C * ap;
  __nv_bfloat16* vhi = alo + C * ap;                                // [C][vp] x 2
  __nv_bfloat16* vlo = vhi + C * vp;
  float* bl = reinterpret_cast<float*>(vhi);                        // GLA, until the values arrive: [C][dimp], [C][rank]
  float* low = bl + C * p.dimp;
  __shared__ float li[C], F[C], G[C], den[C], inter[C], ssum[C][2];
  __shared__ int unsafe[NSUB];
  if (tid < NSUB) unsafe[tid] = 0;
  pi_grid_dependency_wait();
  float m_in = 0.f;
  if (KIND == PI_REC_GLA) {
    gla_decays(p, at, head, low, bl, tot);
    for (int i = tid; i < NSUB * p.dimp; i += kChunkThreads)
      if (tot[i] < kSafeDecay) unsafe[i / p.dimp] = 1;
    // factors between subchunks J <= I (row I (I + 1) / 2 + J), then from the chunk's start to subchunk I
    for (int i = tid; i < kFactors * p.dimp; i += kChunkThreads) {
      const int row = i / p.dimp, d = i - row * p.dimp;
      int I = 0, J = row;
      if (row < kFactors - NSUB) {
        while (J > I) J -= ++I;
      } else {
        I = row - (kFactors - NSUB);
        J = -1;
      }
      float e = I == J ? -tot[I * p.dimp + d] : 0.f;
      for (int x = J + 1; x < I; ++x) e += tot[x * p.dimp + d];
      fac[i] = expf(I == J ? fminf(e, -kSafeDecay) : e);            // beyond: summed pair by pair
    }
  } else {
    mlstm_gates(p, at, head, li, F, G);
    m_in = p.m_in[ch];
    if (tid < C) {
      const float m = fmaxf(F[tid] + m_in, G[tid]);
      inter[tid] = expf(F[tid] + m_in - m);
      den[tid] = m;                                                 // m until the weights are built
    }
    if (tid == 0 && p.chunks[2 * chunk + 1] + C >= p.seq_n[at.seq]) {
      float* st = r.state + (size_t)p.slot[at.seq] * r.state_stride + r.state_off;
      st[(size_t)r.heads * r.dim * r.vdim + (size_t)r.heads * r.dim + head] = fmaxf(F[C - 1] + m_in, G[C - 1]);
    }
  }
  const float* src = p.proj + (size_t)at.row0 * p.stride + (size_t)head * r.dim;
  staged(p.proj, src + r.col_q, p.stride, C, p.dimp, at.n, r.dim, p.vec_k,
         [&](int t, int d, float4 v) {
           float4 e = make_float4(r.q_scale, r.q_scale, r.q_scale, r.q_scale);
           if (KIND == PI_REC_GLA) {
             const float4 b = *reinterpret_cast<const float4*>(bl + t * p.dimp + d);
             e = make_float4(e.x * expf(b.x), e.y * expf(b.y), e.z * expf(b.z), e.w * expf(b.w));
           }
           *reinterpret_cast<float4*>(qf + t * qp + d) = make_float4(v.x * e.x, v.y * e.y, v.z * e.z, v.w * e.w);
         });
  staged(p.proj, src + r.col_k, p.stride, C, p.dimp, at.n, r.dim, p.vec_k,
         [&](int t, int d, float4 v) {
           if (KIND == PI_REC_GLA) {
             const float4 b = *reinterpret_cast<const float4*>(bl + t * p.dimp + d), e = *reinterpret_cast<const float4*>(tot + (t / SUB) * p.dimp + d);
             v = make_float4(v.x * expf(e.x - b.x), v.y * expf(e.y - b.y), v.z * expf(e.z - b.z), v.w * expf(e.w - b.w));
           }
           store_split4(khi, klo, t * kp + d, v);
         });
  __syncthreads();

  // A fragments of 16 query rows at k step ks, GLA: times a factor per channel
  auto q_frag = [&](int row0, int ks, const float* factor, uint32_t* hi, uint32_t* lo) {
    const int rr = row0 + (lane >> 2), c = ks * 16 + (lane & 3) * 2;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int cc = c + (j >> 1) * 8;
      float2 v = *reinterpret_cast<const float2*>(qf + (rr + (j & 1) * 8) * qp + cc);
      if (KIND == PI_REC_GLA) {
        const float2 f = *reinterpret_cast<const float2*>(factor + cc);
        v = make_float2(v.x * f.x, v.y * f.y);
      }
      split(v.x, v.y, hi[j], lo[j]);
    }
  };

  // ---- weights inside the chunk, 16 x 16 tokens at a time ---------------------------------------------------------------
  for (int item = warp; item < NSUB * (NSUB + 1) / 2; item += kChunkWarps) {
    int I = 0, J = item;
    while (J > I) J -= ++I;
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const bool by_pair = KIND == PI_REC_GLA && I == J && unsafe[I];
    if (!by_pair) {
#pragma unroll 1
      for (int ks = 0; ks < nks; ++ks) {
        uint32_t qh[4], ql[4], bh[4], bo[4];
        q_frag(I * SUB, ks, fac + item * p.dimp, qh, ql);
        const int br = J * SUB + (lane & 7) + ((lane >> 4) << 3), bc = ks * 16 + ((lane >> 3) & 1) * 8;
        ldsm4(bh, smem_addr(khi + br * kp + bc));
        ldsm4(bo, smem_addr(klo + br * kp + bc));
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          mma(acc[j], qh[0], qh[1], qh[2], qh[3], bh[2 * j], bh[2 * j + 1]);
          mma(acc[j], ql[0], ql[1], ql[2], ql[3], bh[2 * j], bh[2 * j + 1]);
          mma(acc[j], qh[0], qh[1], qh[2], qh[3], bo[2 * j], bo[2 * j + 1]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = I * SUB + (lane >> 2) + (i >> 1) * 8, s = J * SUB + j * 8 + (lane & 3) * 2 + (i & 1);
        float a = 0.f;
        if (s <= t && t < at.n) {
          if (by_pair) {
            const float* xt = p.proj + (size_t)(at.row0 + t) * p.stride + (size_t)head * r.dim + r.col_q;
            const float* xs = p.proj + (size_t)(at.row0 + s) * p.stride + (size_t)head * r.dim + r.col_k;
            for (int d = 0; d < r.dim; ++d) a = fmaf(xt[d] * r.q_scale * expf(bl[t * p.dimp + d] - bl[s * p.dimp + d]), xs[d], a);
          } else {
            a = acc[j][i];
            if (KIND == PI_REC_MLSTM) a *= expf(F[t] - F[s] + li[s] - den[t]);
          }
        }
        store_split(ahi, alo, t * ap + s, a);
      }
  }
  __syncthreads();
  if (KIND == PI_REC_MLSTM) {   // four threads per token: n_t . q_t
    const int t = tid >> 2, x = tid & 3;
    const float* n_in = p.nU + ch * r.dim;
    float a = 0.f, b = 0.f;
    for (int s = x; s <= t; s += 4) a += __bfloat162float(ahi[t * ap + s]) + __bfloat162float(alo[t * ap + s]);
    for (int d = x; d < r.dim; d += 4) b = fmaf(qf[t * qp + d], n_in[d], b);
    const float dot = quad_sum(fmaf(inter[t], b, a)), m = den[t];
    __syncwarp();
    if (x == 0) den[t] = fmaxf(fabsf(dot), expf(-m)) + 1e-6f;
  }

  // ---- O = Q~ S + A V, 64 value columns at a time; warp = (16 rows, half of the columns) ------------------------------------
  const int I = warp >> 1, half = warp & 1;
  float o[NS][4][4];
  float ss[2] = {0.f, 0.f};
#pragma unroll
  for (int sl = 0; sl < NS; ++sl) {
    const int c0 = sl * kVS;
    __syncthreads();            // the last slice (or the decays in its place) has been read
    load_v(p, at, head, c0, kVS, vhi, vlo, vp);
    const float* S = p.U + ch * r.dim * r.vdim;
    staged(p.proj, S + c0, r.vdim, p.dimp, kVS, r.dim, r.vdim - c0, p.vec_v, [&](int d, int e, float4 v) { store_split4(shi, slo, d * vp + e, v); });
    __syncthreads();
    float (&acc)[4][4] = o[sl];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
    auto products = [&](const uint32_t* ah, const uint32_t* al, const __nv_bfloat16* hi, const __nv_bfloat16* lo, int k0) {
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        uint32_t bh[4], bo[4];
        const int br = k0 + (lane & 7) + ((lane >> 3) & 1) * 8, bc = half * 32 + j * 8 + (lane >> 4) * 8;
        ldsm4_t(bh, smem_addr(hi + br * vp + bc));
        ldsm4_t(bo, smem_addr(lo + br * vp + bc));
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          mma(acc[j + x], ah[0], ah[1], ah[2], ah[3], bh[2 * x], bh[2 * x + 1]);
          mma(acc[j + x], al[0], al[1], al[2], al[3], bh[2 * x], bh[2 * x + 1]);
          mma(acc[j + x], ah[0], ah[1], ah[2], ah[3], bo[2 * x], bo[2 * x + 1]);
        }
      }
    };
#pragma unroll 1
    for (int ks = 0; ks < nks; ++ks) {
      uint32_t qh[4], ql[4];
      q_frag(I * SUB, ks, fac + (kFactors - NSUB + I) * p.dimp, qh, ql);
      products(qh, ql, shi, slo, ks * 16);
    }
    if (KIND == PI_REC_MLSTM) {
      const float f0 = inter[I * SUB + (lane >> 2)], f1 = inter[I * SUB + (lane >> 2) + 8];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[j][0] *= f0;
        acc[j][1] *= f0;
        acc[j][2] *= f1;
        acc[j][3] *= f1;
      }
    }
#pragma unroll 1
    for (int J = 0; J <= I; ++J) {
      uint32_t ah[4], al[4];
      const int ar = I * SUB + (lane & 7) + ((lane >> 3) & 1) * 8, ac = J * SUB + (lane >> 4) * 8;
      ldsm4(ah, smem_addr(ahi + ar * ap + ac));
      ldsm4(al, smem_addr(alo + ar * ap + ac));
      products(ah, al, vhi, vlo, J * SUB);
    }
    if (KIND == PI_REC_MLSTM) {
      const float f0 = 1.f / den[I * SUB + (lane >> 2)], f1 = 1.f / den[I * SUB + (lane >> 2) + 8];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[j][0] *= f0;
        acc[j][1] *= f0;
        acc[j][2] *= f1;
        acc[j][3] *= f1;
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      ss[0] = fmaf(acc[j][0], acc[j][0], fmaf(acc[j][1], acc[j][1], ss[0]));
      ss[1] = fmaf(acc[j][2], acc[j][2], fmaf(acc[j][3], acc[j][3], ss[1]));
    }
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    ss[h] = quad_sum(ss[h]);
    if ((lane & 3) == 0) ssum[I * SUB + (lane >> 2) + 8 * h][half] = ss[h];
  }
  __syncthreads();
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int t = I * SUB + (lane >> 2) + 8 * h;
    if (t >= at.n) continue;
    const float inv = 1.f / sqrtf((ssum[t][0] + ssum[t][1]) / (float)r.vdim + r.eps);
    const float* g = p.proj + (size_t)(at.row0 + t) * p.stride + r.col_g + (size_t)head * r.vdim;
    __nv_bfloat16* out = p.out + (size_t)(at.row0 + t) * p.out_stride + (size_t)head * r.vdim;
    const float* nw = r.norm + (r.norm_per_head ? (size_t)head * r.vdim : 0);
#pragma unroll
    for (int sl = 0; sl < NS; ++sl) {
      float gv[4][2], wv[4][2];
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int e = min(sl * kVS + half * 32 + j * 8 + (lane & 3) * 2 + i, r.vdim - 1);
          gv[j][i] = __ldg(g + e);
          wv[j][i] = __ldg(nw + e);
        }
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int e = sl * kVS + half * 32 + j * 8 + (lane & 3) * 2 + i;
          if (e >= r.vdim) continue;
          const float gate = r.gate_sigmoid ? pi_sigmoid(gv[j][i]) : gv[j][i] * pi_sigmoid(gv[j][i]);
          out[e] = __float2bfloat16_rn(o[sl][j][2 * h + i] * inv * wv[j][i] * gate);
        }
    }
  }
}

size_t local_smem(const ChunkParams& p) {
  const size_t planes = (size_t)2 * C * (p.dimp + 8 + p.vdimp + 8) * 2;
  return planes + (p.r.kind == PI_REC_GLA ? ((size_t)(C + NSUB) * p.dimp + (size_t)C * p.r.rank) * 4 : 0);
}
size_t output_smem(const ChunkParams& p) {
  const bool gla = p.r.kind == PI_REC_GLA;
  const size_t f32 = ((size_t)C * (p.dimp + 4) + (size_t)(NSUB + (gla ? kFactors : 0)) * p.dimp) * 4;
  const size_t keys = (size_t)4 * std::max(C * (p.dimp + 8), p.dimp * (kVS + 8)), weights = (size_t)4 * C * (C + 8), values = (size_t)4 * C * (kVS + 8);
  return f32 + keys + weights + std::max(values, gla ? (size_t)C * (p.dimp + p.r.rank) * 4 : (size_t)0);
}

cudaError_t grant(pi_ctx* ctx, void (*k)(const ChunkParams), size_t smem, pi_smem_grant& g) {
  if (smem <= g.of(ctx) || smem <= kSmemFree) return cudaSuccess;
  g.of(ctx) = smem;
  return cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

void sizes(ChunkParams& p) {
  p.dimp = (p.r.dim + 15) / 16 * 16;
  p.vdimp = (p.r.vdim + 15) / 16 * 16;
}

template <int KIND>
pi_status launch_chunks(pi_ctx* ctx, ChunkParams& p, int n_chunks, int n_seqs) {
  static pi_smem_grant g1, g2[3];
  const pi_recurrence& r = p.r;
  const size_t s1 = local_smem(p), s2 = output_smem(p);
  PI_CUDA(ctx, grant(ctx, recur_local_kernel<KIND>, s1, g1));
  const int passes = (p.vdimp + kVS - 1) / kVS, pick = passes <= 1 ? 0 : passes <= 2 ? 1 : 2;
  void (*const output[3])(const ChunkParams) = {recur_output_kernel<KIND, 1>, recur_output_kernel<KIND, 2>, recur_output_kernel<KIND, 4>};
  PI_CUDA(ctx, grant(ctx, output[pick], s2, g2[pick]));
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, recur_local_kernel<KIND>, dim3(n_chunks, r.heads), dim3(kChunkThreads), s1, 1, p));
  const int per_head = r.dim * r.vdim;
  const bool vec = r.vdim % 4 == 0 && r.state_off % 4 == 0 && r.state_stride % 4 == 0;
  const int elem_blocks = (per_head / (vec ? 4 : 1) + 255) / 256, n_blocks = KIND == PI_REC_MLSTM ? (r.dim + 255) / 256 : 0;
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, vec ? recur_pass_kernel<KIND, 4> : recur_pass_kernel<KIND, 1>, dim3(elem_blocks + n_blocks, r.heads, n_seqs),
                                  dim3(256), 0, 1, p, elem_blocks));
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, output[pick], dim3(n_chunks, r.heads), dim3(kChunkThreads), s2, 1, p));
  return PI_OK;
}

}  // namespace

bool pi_recurrence_chunked(const pi_ctx* ctx, const pi_recurrence& r, int compute) {
  ChunkParams p = {};
  p.r = r;
  sizes(p);
  return compute == PI_BF16 && r.dim <= kMaxDim && r.vdim <= kMaxVdim && std::max(local_smem(p), output_smem(p)) + 4096 <= ctx->smem_optin;
}

size_t pi_recurrence_scratch_floats(const pi_recurrence& r, int n_chunks) {
  const size_t per = (size_t)r.dim * r.vdim + 2 * (size_t)r.dim + 8;
  return n_chunks ? (size_t)n_chunks * r.heads * per + 64 : 0;
}

pi_status pi_launch_recurrence_chunks(pi_ctx* ctx, const pi_recurrence& r, const float* proj, size_t stride, __nv_bfloat16* out, size_t out_stride,
                                      const pi_seq_batch& b, float* scratch) {
  ChunkParams p = {};
  p.r = r;
  p.proj = proj;
  p.stride = stride;
  p.out = out;
  p.out_stride = out_stride;
  p.chunk_seqs = b.chunk_seqs;
  p.chunks = b.chunks;
  p.chunk0 = b.chunk0;
  p.seq_row0 = b.seq_row0;
  p.seq_n = b.seq_n;
  p.seq_start = b.seq_start;
  p.slot = b.slot;
  sizes(p);
  p.vec_k = r.dim % 4 == 0 && r.col_q % 4 == 0 && r.col_k % 4 == 0 && stride % 4 == 0;
  p.vec_v = r.vdim % 4 == 0 && r.col_v % 4 == 0 && stride % 4 == 0;
  const size_t ch = (size_t)b.n_chunks * r.heads;
  p.U = scratch;
  p.nU = p.U + (ch * r.dim * r.vdim + 3) / 4 * 4;
  p.decay = p.nU + ch * r.dim;
  p.FG = p.decay + ch * r.dim;
  p.m_in = p.FG + 2 * ch;
  return r.kind == PI_REC_GLA ? launch_chunks<PI_REC_GLA>(ctx, p, b.n_chunks, b.n_chunk_seqs)
                              : launch_chunks<PI_REC_MLSTM>(ctx, p, b.n_chunks, b.n_chunk_seqs);
}
