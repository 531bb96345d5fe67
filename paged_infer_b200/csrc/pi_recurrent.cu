// Recurrent token mixers with a matrix state per head, f32 throughout:
//
//   GLA     S_t = diag(a_t) S_(t-1) + k_t v_t^T,  a_t = exp(log_sigmoid(z_t) / tau) per key channel
//           o_t = S_t^T q_t
//   mLSTM   m_t = max(f_t + m_(t-1), i_t)
//           S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T,  n_t likewise with k_t alone
//           o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6)
//   then    out = o / rms(o) * norm * gate(g)     per head
//
// recur_scan_kernel walks the tokens of a sequence one by one with the state in registers: the decode kernel, and the
// one that takes short portions.  A head's value channels are cut into slices of 128 columns; the CTAs of a head form
// a thread-block cluster, which adds up the head's sum of squares through distributed shared memory and keeps the
// shared n and m consistent (everybody reads them before anybody writes).  For key sizes whose state does not fit the
// registers it stays in global memory (R = 0).  Long portions take the kernels of pi_recurrent_chunk.cu.
#include <cooperative_groups.h>
#include <math.h>

#include <algorithm>

#include "pi_layered.cuh"

namespace cg = cooperative_groups;

namespace {

constexpr int kWarps = 8;
constexpr int kThreads = kWarps * 32;
constexpr int kSlice = 128;        // value columns of a CTA: four per lane
constexpr int kMaxSlices = 8;      // portable cluster size

struct RecParams {
  pi_recurrence r;
  const float* proj;
  size_t stride;
  void* out;
  size_t out_stride;
  const int32_t *seqs, *seq_row0, *seq_n, *seq_start, *slot;
  int slices, vec;
};

__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }

// Sum over the CTA's threads, the same bits in every thread.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = pi_warp_sum(v);
  __syncthreads();                    // red may still be read from the last call
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) t += red[w];
  return t;
}

// R > 0: each warp keeps rows w, w + 8, ... (R of them) of the slice in registers.  R == 0: state in global memory.
template <int KIND, int R, typename O>
__global__ void __launch_bounds__(kThreads) recur_scan_kernel(const RecParams p) {
  extern __shared__ float sm[];
  const pi_recurrence& r = p.r;
  float* sq = sm;                    // [dim]
  float* sk = sq + r.dim;            // [dim]
  float* sa = sk + r.dim;            // [dim] decay per channel (GLA)
  float* slow = sa + r.dim;          // [rank] low-rank gate input (GLA)
  float* part = sm + ((3 * r.dim + r.rank + 3) & ~3);   // [warps][kSlice]
  __shared__ float red[kWarps];
  __shared__ float s_ss[2];          // sum of squares of this slice, by token parity (read by the cluster)
  const int slice = blockIdx.x, head = blockIdx.y, seq = p.seqs[blockIdx.z];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int row0 = p.seq_row0[seq], n_tok = p.seq_n[seq];
  const bool fresh = p.seq_start[seq] == 0;
  float* st = r.state + (size_t)p.slot[seq] * r.state_stride + r.state_off;
  float* S = st + (size_t)head * r.dim * r.vdim;
  float* nst = st + (size_t)r.heads * r.dim * r.vdim + (size_t)head * r.dim;
  float* mst = st + (size_t)r.heads * r.dim * r.vdim + (size_t)r.heads * r.dim + head;
  const int e0 = slice * kSlice + lane * 4;
  const bool vec = p.vec != 0;
  const int nv = min(4, r.vdim - e0);   // columns of this lane that exist (may be <= 0)

  auto load4 = [&](const float* src) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (vec) {
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
    if (vec) {
      if (nv > 0) *reinterpret_cast<float4*>(dst) = v;
    } else {
      if (nv > 0) dst[0] = v.x;
      if (nv > 1) dst[1] = v.y;
      if (nv > 2) dst[2] = v.z;
      if (nv > 3) dst[3] = v.w;
    }
  };

  // the state was written by an earlier step: it may be read ahead of the dependency wait
  float4 s[R > 0 ? R : 1];
  if (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int d = warp + i * kWarps;
      s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && d < r.dim) s[i] = load4(S + (size_t)d * r.vdim + e0);
    }
  }
  float nreg[4] = {0.f, 0.f, 0.f, 0.f}, m = 0.f;   // mLSTM: n of channels tid, tid + 256, ... (up to 1024)
  if (KIND == PI_REC_MLSTM && !fresh) {
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (tid + j * kThreads < r.dim) nreg[j] = nst[tid + j * kThreads];
    m = *mst;
  }
  pi_grid_dependency_wait();
  if (p.slices > 1) cg::this_cluster().sync();     // every slice has read n and m before slice 0 writes them

  for (int t = 0; t < n_tok; ++t) {
    const float* x = p.proj + (size_t)(row0 + t) * p.stride;
    const float4 v = load4(x + r.col_v + (size_t)head * r.vdim + e0);
    __syncthreads();                               // the last token's readers of sq / sk / sa are done
    for (int d = tid; d < r.dim; d += kThreads) {
      sq[d] = x[r.col_q + (size_t)head * r.dim + d] * r.q_scale;
      sk[d] = x[r.col_k + (size_t)head * r.dim + d];
    }
    float keep = 1.f, put = 1.f, floor_m = 0.f;
    if (KIND == PI_REC_GLA) {
      for (int j = tid; j < r.rank; j += kThreads) slow[j] = x[r.col_low + j];
      __syncthreads();
      for (int d = tid; d < r.dim; d += kThreads) {
        const int c = head * r.dim + d;
        const float* w = r.a2 + (size_t)c * r.rank;
        float z = 0.f;
        for (int j = 0; j < r.rank; ++j) z = fmaf(w[j], slow[j], z);
        sa[d] = expf(pi_log_sigmoid(z + r.a2_b[c]) / r.tau);
      }
    } else {
      const float li = soft_cap(x[r.col_i + head] + r.i_b[head], r.gate_cap);
      const float lf = pi_log_sigmoid(soft_cap(x[r.col_f + head] + r.f_b[head], r.gate_cap));
      const float mn = fmaxf(lf + m, li);
      keep = expf(lf + m - mn);
      put = expf(li - mn);
      floor_m = expf(-mn);
      m = mn;
    }
    __syncthreads();
    float den = 1.f;
    if (KIND == PI_REC_MLSTM) {
      float dot = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int d = tid + j * kThreads;
        if (d < r.dim) {
          nreg[j] = fmaf(keep, nreg[j], put * sk[d]);
          dot = fmaf(nreg[j], sq[d], dot);
        }
      }
      den = fmaxf(fabsf(block_sum(dot, red)), floor_m) + 1e-6f;
    }
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    auto step = [&](float4& sv, int d) {
      const float a = KIND == PI_REC_GLA ? sa[d] : keep;
      const float kk = KIND == PI_REC_GLA ? sk[d] : put * sk[d];
      const float qq = sq[d];
      sv.x = fmaf(a, sv.x, kk * v.x);
      sv.y = fmaf(a, sv.y, kk * v.y);
      sv.z = fmaf(a, sv.z, kk * v.z);
      sv.w = fmaf(a, sv.w, kk * v.w);
      o.x = fmaf(sv.x, qq, o.x);
      o.y = fmaf(sv.y, qq, o.y);
      o.z = fmaf(sv.z, qq, o.z);
      o.w = fmaf(sv.w, qq, o.w);
    };
    if (R > 0) {
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int d = warp + i * kWarps;
        if (d < r.dim) step(s[i], d);
      }
    } else {
      for (int d = warp; d < r.dim; d += kWarps) {
        float4 sv = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!(fresh && t == 0)) sv = load4(S + (size_t)d * r.vdim + e0);
        step(sv, d);
        store4(S + (size_t)d * r.vdim + e0, sv);
      }
    }
    *reinterpret_cast<float4*>(part + warp * kSlice + lane * 4) = o;
    __syncthreads();
    const int e = slice * kSlice + tid;
    const bool mine = tid < kSlice && e < r.vdim;
    float ov = 0.f;
    if (mine) {
#pragma unroll
      for (int w = 0; w < kWarps; ++w) ov += part[w * kSlice + tid];
      if (KIND == PI_REC_MLSTM) ov /= den;
    }
    float ss = block_sum(mine ? ov * ov : 0.f, red);
    if (p.slices > 1) {                            // the head's sum of squares, added in slice order
      cg::cluster_group cl = cg::this_cluster();
      if (tid == 0) s_ss[t & 1] = ss;
      cl.sync();
      ss = 0.f;
      for (int c = 0; c < p.slices; ++c) ss += *cl.map_shared_rank(&s_ss[t & 1], c);
    }
    if (mine) {
      const int c = head * r.vdim + e;
      const float g = x[r.col_g + c];
      const float gate = r.gate_sigmoid ? pi_sigmoid(g) : g * pi_sigmoid(g);
      const float y = ov / sqrtf(ss / (float)r.vdim + r.eps) * r.norm[r.norm_per_head ? c : e] * gate;
      static_cast<O*>(p.out)[(size_t)(row0 + t) * p.out_stride + c] = pi_from_f32<O>(y);
    }
  }

  if (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int d = warp + i * kWarps;
      if (d < r.dim) store4(S + (size_t)d * r.vdim + e0, s[i]);
    }
  }
  if (KIND == PI_REC_MLSTM && slice == 0) {
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (tid + j * kThreads < r.dim) nst[tid + j * kThreads] = nreg[j];
    if (tid == 0) *mst = m;
  }
  if (p.slices > 1) cg::this_cluster().sync();     // a peer may still be reading this CTA's sum of squares
}

template <int KIND, typename O>
void (*pick_scan(int dim))(const RecParams) {
  const int need = (dim + kWarps - 1) / kWarps;
  if (need <= 4) return recur_scan_kernel<KIND, 4, O>;
  if (need <= 8) return recur_scan_kernel<KIND, 8, O>;
  if (need <= 16) return recur_scan_kernel<KIND, 16, O>;
  if (need <= 32) return recur_scan_kernel<KIND, 32, O>;
  return recur_scan_kernel<KIND, 0, O>;
}

}  // namespace

pi_status pi_launch_recurrence(pi_ctx* ctx, const pi_recurrence& r, const float* proj, size_t stride, void* out, size_t out_stride,
                               int out_kind, const pi_seq_batch& b, float* scratch) {
  pi_prof_scope prof(ctx, PI_PROF_RECURRENCE);
  const int slices = (r.vdim + kSlice - 1) / kSlice;
  PI_REQUIRE(ctx, slices <= kMaxSlices && r.dim <= 1024, "recurrent heads of %d x %d channels are not supported (at most 1024 x %d)", r.dim,
             r.vdim, kMaxSlices * kSlice);
  if (b.n_scan > 0) {
    RecParams p = {r, proj, stride, out, out_stride, b.scan_seqs, b.seq_row0, b.seq_n, b.seq_start, b.slot, slices, 0};
    p.vec = r.vdim % 4 == 0 && r.col_v % 4 == 0 && stride % 4 == 0 && r.state_off % 4 == 0 && r.state_stride % 4 == 0;
    void (*k)(const RecParams);
    if (r.kind == PI_REC_GLA) k = out_kind == PI_BF16 ? pick_scan<PI_REC_GLA, __nv_bfloat16>(r.dim) : pick_scan<PI_REC_GLA, float>(r.dim);
    else k = out_kind == PI_BF16 ? pick_scan<PI_REC_MLSTM, __nv_bfloat16>(r.dim) : pick_scan<PI_REC_MLSTM, float>(r.dim);
    const size_t smem = sizeof(float) * ((size_t)3 * r.dim + r.rank + 4 + kWarps * kSlice);
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(slices, r.heads, b.n_scan), dim3(kThreads), smem, slices, p));
  }
  if (b.n_chunks > 0) {
    PI_REQUIRE(ctx, out_kind == PI_BF16 && scratch, "long portions run on the tensor-core path");
    return pi_launch_recurrence_chunks(ctx, r, proj, stride, static_cast<__nv_bfloat16*>(out), out_stride, b, scratch);
  }
  return PI_OK;
}
