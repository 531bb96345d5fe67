// Tensor-core GEMM for bf16 weights and bf16 activations: out[m][n] = sum_k W[n][k] x[m][k], f32 accumulation in tensor
// memory, with the epilogues of the layered designs.
//
// As in pi_gemm_tc.cu the weight rows sit on the MMA's M axis (128 TMEM lanes per tile) and the activation rows on its N
// axis (16..256 columns), so that one kernel serves decode batches and prefill.  Both operands arrive by TMA (64 K
// elements per stage, 128-byte swizzle; anything past K, N or M reads as zero, so sizes need not be multiples of the
// tile).  A thread of the epilogue owns one output column n and walks the rows m: the 32 lanes of a warp store 32
// adjacent columns of one row.
//
// Warps 0-7: epilogue; warp 8: TMA; warp 9: tensor memory and MMA issue.  Launches with enough tiles are persistent (one CTA
// per SM, two accumulators: the epilogue of a tile overlaps the products of the next).  Launches with few tiles split
// K over a thread-block cluster: every CTA parks its partial tile in shared memory and finishes every ksplit-th column,
// adding the slices in rank order.  Weight tiles of the first stages are requested before the dependency wait.  All
// waits are bounded; one that runs out sets the context's error word.
//
// GROUPED: the weights are a stack of experts and the activation rows lie grouped by expert; a device-built table names the
// column tiles (expert, first row, rows), so that the launch needs no routing result on the host.  Every tile is
// multiplied in full; what belongs to the next expert is dropped in the epilogue.
#include <cooperative_groups.h>

#include <algorithm>

#include "pi_gemm_tc.cuh"
#include "pi_layered.cuh"

namespace cg = cooperative_groups;

namespace {
using pi_tc::mbar_arrive;
using pi_tc::mbar_arrive_expect_tx;
using pi_tc::mbar_init;
using pi_tc::mbar_wait_dep;
using pi_tc::smem_desc;
using pi_tc::smem_u32;
using pi_tc::tmem_ld16_issue;
using pi_tc::umma_commit;

constexpr int kTM = 128;            // weight rows per tile
constexpr int kTK = 64;             // K elements per stage: one 128-byte swizzle atom
constexpr int kEpiWarps = 8;
constexpr int kGemmThreads = (kEpiWarps + 2) * 32;
constexpr int kTmemCols = 512;      // all columns: two of these CTAs never share an SM (see pi_gemm_tc.cuh)
constexpr size_t kMinSmemBytes = 120 * 1024;

struct Bf16GemmParams {
  float* out;
  __nv_bfloat16* out_bf16;
  size_t out_stride;
  int N, K, M, nkb, rtiles, tiles, ksplit, epi;   // N: of one expert
  pi_dyt_residual res;
  pi_maps_kv mkv;
  const float* out_scale;
  pi_token_table table;
  float glu_limit;
  int glu_rows;
  float* rest;
  size_t rest_stride;
  const int4* tile_table;         // GROUPED
  const int32_t* n_tiles;
  int* err_flag;
};

// A column tile: which expert, its activation rows [m0, m_end).
struct TileAt {
  int expert, m0, m_end;
};

__device__ __forceinline__ void umma_f16_ss(uint32_t tmem_d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(tmem_d), "l"(a), "l"(b), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void tma_2d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int x, int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];" ::"r"(dst), "l"(map), "r"(bar),
      "r"(x), "r"(y)
      : "memory");
}

// C columns (activation rows m, m + dm, ... < M) of output column n, all lanes of the warp on adjacent n.  `place`: of row m, if
// it has been looked up already.
template <int C>
__device__ __forceinline__ void epilogue(const Bf16GemmParams& p, int M, int n, int m, int dm, const float* v, const pi_kv_place* place = nullptr) {
  const bool ok = n < p.N;
  if (p.epi == PI_EPI_DYT_RESIDUAL) {
    float old[C];
#pragma unroll
    for (int j = 0; j < C; ++j) old[j] = (ok && m + j * dm < M) ? p.res.x[(size_t)(m + j * dm) * p.res.x_stride + n] : 0.f;
    const float wp = ok ? __ldg(p.res.post.w + n) : 0.f, bp = ok ? __ldg(p.res.post.b + n) : 0.f;
    const float wn = ok ? __ldg(p.res.next.w + n) : 0.f, bn = ok ? __ldg(p.res.next.b + n) : 0.f;
#pragma unroll
    for (int j = 0; j < C; ++j) {
      if (!ok || m + j * dm >= M) continue;
      const float x = old[j] + fmaf(tanhf(p.res.post.alpha * v[j]), wp, bp);
      p.res.x[(size_t)(m + j * dm) * p.res.x_stride + n] = x;
      static_cast<__nv_bfloat16*>(p.res.h)[(size_t)(m + j * dm) * p.res.h_stride + n] =
          __float2bfloat16_rn(fmaf(tanhf(p.res.next.alpha * x), wn, bn));
    }
  } else if (p.epi == PI_EPI_MAPS_QKV) {
    // a rotation pair is two adjacent columns, so the partner is the neighbouring lane; lane j looks row j's place up
    const pi_maps_kv& k = p.mkv;
    const pi_maps_col col = pi_maps_column(k, min(n, p.N - 1));
    const int lane = threadIdx.x & 31;
    pi_kv_place mine = {0, -1, 0};
    const int my_row = m + (C == 1 ? 0 : (lane % C) * dm);
    if (place) mine = *place;
    else if (my_row < M) mine = pi_maps_kv_place(k, my_row);
    const int half = k.rot_dims >> 1, pair = col.rotated ? col.d >> 1 : 0;
    float cs[C], sn[C];
    if (half > 0) {
#pragma unroll
      for (int j = 0; j < C; ++j) {
        const size_t at = (size_t)__shfl_sync(0xffffffffu, mine.pos, j) * half + pair;
        cs[j] = __ldg(k.rope_cos + at);
        sn[j] = __ldg(k.rope_sin + at);
      }
    }
    const float bias = k.bias ? __ldg(k.bias + min(n, p.N - 1)) : 0.f;
#pragma unroll
    for (int j = 0; j < C; ++j) {
      float r = v[j] + bias;
      const float other = __shfl_xor_sync(0xffffffffu, r, 1);
      const int pos = __shfl_sync(0xffffffffu, mine.pos, j), block = __shfl_sync(0xffffffffu, mine.block, j), off = __shfl_sync(0xffffffffu, mine.off, j);
      if (col.rotated) r = (n & 1) ? r * cs[j] + other * sn[j] : r * cs[j] - other * sn[j];
      if (!ok || m + j * dm >= M) continue;
      r = pi_maps_finish(k, col, m + j * dm, n, pos, r);
      if (col.is_q) p.out[(size_t)(m + j * dm) * p.out_stride + n] = r;
      else pi_maps_kv_store(k, col, block, off, r);
    }
  } else if (p.epi == PI_EPI_GEGLU || p.epi == PI_EPI_SWIGLU || p.epi == PI_EPI_CLAMP_GLU) {
    // even n: gate rows, odd n: up rows; of two columns m the even lane finishes the first, the odd lane the second
    const int odd = n & 1;
    const bool pair = n < p.glu_rows;
    if (C == 1) {
      const float other = __shfl_xor_sync(0xffffffffu, v[0], 1);
      if (pair && !odd && m < M) p.out_bf16[(size_t)m * p.out_stride + (n >> 1)] = __float2bfloat16_rn(pi_glu(p.epi, v[0], other, p.glu_limit));
    } else {
#pragma unroll
      for (int j = 0; j + 1 < C; j += 2) {
        const float other = __shfl_xor_sync(0xffffffffu, odd ? v[j] : v[j + 1], 1);
        const float g = odd ? other : v[j], u = odd ? v[j + 1] : other;
        const int mm = m + (j + odd) * dm;
        if (pair && mm < M) p.out_bf16[(size_t)mm * p.out_stride + (n >> 1)] = __float2bfloat16_rn(pi_glu(p.epi, g, u, p.glu_limit));
      }
    }
    if (ok && !pair) {
#pragma unroll
      for (int j = 0; j < C; ++j)
        if (m + j * dm < M) p.rest[(size_t)(m + j * dm) * p.rest_stride + (n - p.glu_rows)] = v[j];
    }
  } else if (p.epi == PI_EPI_SCALE_ADD) {
    float old[C];
#pragma unroll
    for (int j = 0; j < C; ++j) old[j] = (ok && m + j * dm < M) ? p.out[(size_t)(m + j * dm) * p.out_stride + n] : 0.f;
    const float w = ok ? __ldg(p.out_scale + n) : 0.f;
#pragma unroll
    for (int j = 0; j < C; ++j)
      if (ok && m + j * dm < M) p.out[(size_t)(m + j * dm) * p.out_stride + n] = fmaf(w, v[j], old[j]);
  } else if (p.epi == PI_EPI_GELU_TABLE) {
    float e[C];
#pragma unroll
    for (int j = 0; j < C; ++j) e[j] = pi_table_value(p.table, min(m + j * dm, M - 1), min(n, p.N - 1));
#pragma unroll
    for (int j = 0; j < C; ++j)
      if (ok && m + j * dm < M) p.out_bf16[(size_t)(m + j * dm) * p.out_stride + n] = __float2bfloat16_rn(pi_gelu_tanh(v[j]) * e[j]);
  } else if (p.epi == PI_EPI_RELU2) {
#pragma unroll
    for (int j = 0; j < C; ++j) {
      const float r = fmaxf(v[j], 0.f);
      if (ok && m + j * dm < M) p.out_bf16[(size_t)(m + j * dm) * p.out_stride + n] = __float2bfloat16_rn(r * r);
    }
  } else if (p.out_bf16) {
#pragma unroll
    for (int j = 0; j < C; ++j)
      if (ok && m + j * dm < M) p.out_bf16[(size_t)(m + j * dm) * p.out_stride + n] = __float2bfloat16_rn(v[j]);
  } else {
#pragma unroll
    for (int j = 0; j < C; ++j)
      if (ok && m + j * dm < M) p.out[(size_t)(m + j * dm) * p.out_stride + n] = v[j];
  }
}

template <int BN, int STAGES, bool SPLIT, bool GROUPED = false>
__global__ void __launch_bounds__(kGemmThreads, 1)
gemm_bf16_kernel(const Bf16GemmParams p, const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x) {
  constexpr int kABytes = kTM * kTK * 2, kBBytes = BN * kTK * 2, kStageBytes = kABytes + kBBytes;
  constexpr int kAcc = SPLIT ? 1 : 2;
  static_assert(kAcc * BN <= kTmemCols, "accumulators exceed tensor memory");
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) unsigned long long bars[2 * STAGES + 4];
  __shared__ uint32_t s_tmem;
  __shared__ volatile int s_abort, s_dep_ok;
  __shared__ pi_kv_place s_place[SPLIT ? BN : 1];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t full0 = smem_u32(&bars[0]), empty0 = smem_u32(&bars[STAGES]), acc_full0 = smem_u32(&bars[2 * STAGES]),
                 acc_empty0 = smem_u32(&bars[2 * STAGES + 2]);
  const uint32_t base = smem_u32(smem);
  // this CTA's tiles and its K blocks
  const int rank = SPLIT ? (int)blockIdx.x % p.ksplit : 0;
  const int tile0 = SPLIT ? (int)blockIdx.x / p.ksplit : (int)blockIdx.x, tile_step = SPLIT ? p.tiles : (int)gridDim.x;
  const int kb0 = SPLIT ? (int)((long)rank * p.nkb / p.ksplit) : 0, kb1 = SPLIT ? (int)((long)(rank + 1) * p.nkb / p.ksplit) : p.nkb;
  const int nk = kb1 - kb0;
  static_assert(!(SPLIT && GROUPED), "the table's length is not known when the launch is cut");
  auto count = [&](int tiles) { return tile0 < tiles ? (tiles - tile0 + tile_step - 1) / tile_step : 0; };
  int my_tiles = GROUPED ? 0 : count(p.tiles);   // GROUPED: every role reads it behind its own wait
  auto tile_at = [&](int tile) {
    TileAt t = {0, (tile / p.rtiles) * BN, p.M};
    if (GROUPED) {
      const int4 e = p.tile_table[tile / p.rtiles];
      t.expert = e.x;
      t.m0 = e.y;
      t.m_end = e.y + e.z;
    }
    return t;
  };

  if (tid == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(full0 + 8 * s, 1);
      mbar_init(empty0 + 8 * s, 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(acc_full0 + 8 * a, 1);
      mbar_init(acc_empty0 + 8 * a, kEpiWarps);
    }
    s_abort = 0;
    s_dep_ok = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == kEpiWarps + 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(kTmemCols));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  pi_grid_launch_dependents();   // only now that this CTA holds its tensor memory
  const uint32_t tmem = s_tmem;

  auto give_up = [&](int code) {
    if (!s_abort && p.err_flag) atomicExch(p.err_flag, code);
    s_abort = 1;
  };

  if (warp == kEpiWarps) {
    // ---- TMA ------------------------------------------------------------------------------------------------------
    if (lane == 0) {
      if (GROUPED) {
        pi_grid_dependency_wait();
        s_dep_ok = 1;
        my_tiles = count(*p.n_tiles * p.rtiles);
      }
      const int total = my_tiles * nk;
      auto load_w = [&](int it) {
        const int tile = tile0 + (it / nk) * tile_step, kb = kb0 + it % nk, s = it % STAGES;
        mbar_arrive_expect_tx(full0 + 8 * s, kStageBytes);
        tma_2d(base + s * kStageBytes, &map_w, full0 + 8 * s, kb * kTK, (GROUPED ? tile_at(tile).expert * p.N : 0) + (tile % p.rtiles) * kTM);
      };
      auto load_x = [&](int it) {
        const int tile = tile0 + (it / nk) * tile_step, kb = kb0 + it % nk, s = it % STAGES;
        tma_2d(base + s * kStageBytes + kABytes, &map_x, full0 + 8 * s, kb * kTK, tile_at(tile).m0);
      };
      const int ahead = min(total, STAGES);
      for (int it = 0; it < ahead; ++it) load_w(it);   // weights never depend on the preceding kernel
      if (!GROUPED) pi_grid_dependency_wait();
      s_dep_ok = 1;
      for (int it = 0; it < ahead; ++it) load_x(it);
      int issued = ahead;
      for (int it = ahead; it < total; ++it, ++issued) {
        if (s_abort || !mbar_wait_dep(empty0 + 8 * (it % STAGES), ((it / STAGES) & 1) ^ 1, &s_dep_ok)) {
          give_up(21);
          break;
        }
        load_w(it);
        load_x(it);
      }
      if (s_abort)   // no copy of this CTA may still be in flight when it leaves
        for (int it = max(0, issued - STAGES); it < issued; ++it) pi_tc::mbar_wait(full0 + 8 * (it % STAGES), (it / STAGES) & 1);
    }
  } else if (warp == kEpiWarps + 1) {
    // ---- MMA ------------------------------------------------------------------------------------------------------
    if (lane == 0) {
      if (GROUPED) {
        pi_grid_dependency_wait();
        my_tiles = count(*p.n_tiles * p.rtiles);
      }
      const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kTM >> 4) << 24);
      int it = 0;
      bool ok = true;
      for (int t = 0; t < my_tiles && ok; ++t) {
        const int a = t % kAcc;
        if (t >= kAcc && !mbar_wait_dep(acc_empty0 + 8 * a, ((t / kAcc) & 1) ^ 1, &s_dep_ok)) {
          give_up(22);
          break;
        }
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        for (int kb = 0; kb < nk; ++kb, ++it) {
          const int s = it % STAGES;
          if (s_abort || !mbar_wait_dep(full0 + 8 * s, (it / STAGES) & 1, &s_dep_ok)) {
            give_up(23);
            ok = false;
            break;
          }
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          const uint64_t da = smem_desc(base + s * kStageBytes), db = smem_desc(base + s * kStageBytes + kABytes);
#pragma unroll
          for (int ks = 0; ks < kTK / 16; ++ks)
            umma_f16_ss(tmem + a * BN, da + (uint64_t)((ks * 32) >> 4), db + (uint64_t)((ks * 32) >> 4), idesc, (kb | ks) ? 1u : 0u);
          umma_commit(empty0 + 8 * s);
        }
        if (ok) umma_commit(acc_full0 + 8 * a);
      }
    }
  } else {
    // ---- epilogue: warp w reads TMEM lanes 32 (w % 4).., warps 0-3 the first half of the columns, 4-7 the second ----
    const int quad = warp & 3, half = warp >> 2;
    constexpr int kHalfCols = BN >= 32 ? BN / 2 : 16;
    if (SPLIT && p.epi == PI_EPI_MAPS_QKV)   // the rows' places do not depend on the preceding kernel
      for (int c = tid; c < BN && (tile0 / p.rtiles) * BN + c < p.M; c += kEpiWarps * 32)
        s_place[c] = pi_maps_kv_place(p.mkv, (tile0 / p.rtiles) * BN + c);
    pi_grid_dependency_wait();   // the epilogue reads and writes what the preceding kernels use
    if (GROUPED) my_tiles = count(*p.n_tiles * p.rtiles);
    for (int t = 0; t < my_tiles; ++t) {
      const int a = t % kAcc, tile = tile0 + t * tile_step;
      int got = 0;
      if (lane == 0) {
        got = !s_abort && mbar_wait_dep(acc_full0 + 8 * a, (t / kAcc) & 1, &s_dep_ok);
        if (!got) give_up(24);
      }
      got = __shfl_sync(0xffffffffu, got, 0);
      if (!got) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const TileAt at = tile_at(tile);
      const int n = (tile % p.rtiles) * kTM + quad * 32 + lane, m0 = at.m0;
      if (BN >= 32 || half == 0) {
#pragma unroll 1
        for (int c = half * kHalfCols; c < half * kHalfCols + kHalfCols; c += 16) {
          if (!SPLIT && m0 + c >= at.m_end) break;
          uint32_t r[16];
          tmem_ld16_issue(tmem + ((uint32_t)(quad * 32) << 16) + (uint32_t)(a * BN + c), r);
          asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
          float v[16];
#pragma unroll
          for (int j = 0; j < 16; ++j) v[j] = __uint_as_float(r[j]);
          if (SPLIT) {
            float* part = reinterpret_cast<float*>(smem + STAGES * kStageBytes);
#pragma unroll
            for (int j = 0; j < 16; ++j) part[(c + j) * kTM + quad * 32 + lane] = v[j];
          } else {
            epilogue<16>(p, at.m_end, n, m0 + c, 1, v);
          }
        }
      }
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(acc_empty0 + 8 * a);
    }
  }

  if (SPLIT) {
    cg::cluster_group cluster = cg::this_cluster();
    __syncwarp();
    cluster.sync();
    float* part = reinterpret_cast<float*>(smem + STAGES * kStageBytes);
    if (warp < kEpiWarps && !s_abort) {
      const int row = tid & (kTM - 1), n = (tile0 % p.rtiles) * kTM + row, m0 = (tile0 / p.rtiles) * BN;
      for (int c = rank + (tid >> 7) * p.ksplit; c < BN && m0 + c < p.M; c += 2 * p.ksplit) {
        float s[8];
#pragma unroll
        for (int r = 0; r < 8; ++r) s[r] = r < p.ksplit ? cluster.map_shared_rank(part, r)[c * kTM + row] : 0.f;
        float v = 0.f;
#pragma unroll
        for (int r = 0; r < 8; ++r) v += s[r];
        epilogue<1>(p, p.M, n, m0 + c, 1, &v, &s_place[c]);
      }
    }
    __syncwarp();
    cluster.sync();   // nobody leaves while a peer still reads its partial tile
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == kEpiWarps + 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kTmemCols));
  }
}

template <int BN, int STAGES, bool SPLIT>
constexpr size_t gemm_smem() {
  return std::max((size_t)STAGES * (kTM + BN) * kTK * 2 + (SPLIT ? (size_t)BN * kTM * 4 : 0) + 1024, kMinSmemBytes);
}

template <int BN, int STAGES, bool SPLIT, bool GROUPED = false>
cudaError_t launch(pi_ctx* ctx, const Bf16GemmParams& p, const CUtensorMap& w, const CUtensorMap& x, int ctas) {
  auto k = gemm_bf16_kernel<BN, STAGES, SPLIT, GROUPED>;
  constexpr size_t smem = gemm_smem<BN, STAGES, SPLIT>();
  static pi_smem_grant granted;
  if (smem > granted.of(ctx)) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    granted.of(ctx) = smem;
  }
  return pi_launch_dep(ctx, k, dim3(ctas), dim3(kGemmThreads), smem, SPLIT ? p.ksplit : 1, p, w, x);
}

// Clusters of `ksplit` CTAs the device holds at once.
template <int BN, int STAGES>
int max_clusters(pi_ctx* ctx, int ksplit) {
  static int cached[9] = {};
  if (!cached[ksplit]) {
    auto k = gemm_bf16_kernel<BN, STAGES, true>;
    constexpr size_t smem = gemm_smem<BN, STAGES, true>();
    cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(ksplit);
    cfg.blockDim = dim3(kGemmThreads);
    cfg.dynamicSmemBytes = smem;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = ksplit;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    int n = 0;
    if (cudaOccupancyMaxActiveClusters(&n, k, &cfg) != cudaSuccess || n <= 0) {
      cudaGetLastError();
      n = std::max(1, ctx->sm_count / ksplit / 2);
    }
    cached[ksplit] = n;
  }
  return cached[ksplit];
}

template <int BN, int STAGES>
cudaError_t run(pi_ctx* ctx, Bf16GemmParams& p, const CUtensorMap& w, const CUtensorMap& x) {
  if (BN <= 128) {
    for (int ks = 8; ks >= 2; --ks)
      if (p.nkb / ks >= 2 && p.tiles * ks <= ctx->sm_count && p.tiles <= max_clusters<(BN <= 128 ? BN : 128), STAGES>(ctx, ks)) {
        p.ksplit = ks;
        return launch<(BN <= 128 ? BN : 128), STAGES, true>(ctx, p, w, x, p.tiles * ks);
      }
  }
  p.ksplit = 1;
  return launch<BN, STAGES, false>(ctx, p, w, x, std::min(p.tiles, ctx->sm_count));
}
template <int BN, int STAGES>
cudaError_t run_grouped(pi_ctx* ctx, Bf16GemmParams& p, const CUtensorMap& w, const CUtensorMap& x) {
  p.ksplit = 1;
  return launch<BN, STAGES, false, true>(ctx, p, w, x, std::min(p.tiles, ctx->sm_count));
}

pi_status encode_2d(pi_ctx* ctx, CUtensorMap* map, const void* base, size_t cols, size_t rows, size_t ld, int box_rows) {
  const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
  const cuuint32_t box[2] = {kTK, (cuuint32_t)box_rows};
  const cuuint32_t estr[2] = {1, 1};
  const auto fn = pi_tc::encode_tiled_fn();
  PI_REQUIRE(ctx, fn, "cuTensorMapEncodeTiled is not available");
  const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                        CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return pi_fail(ctx, PI_ERR_CUDA, "cuTensorMapEncodeTiled failed with %d", (int)r);
  return PI_OK;
}

}  // namespace

pi_status pi_launch_gemm_bf16(pi_ctx* ctx, const pi_linear* lin, const pi_linear_args& a) {
  PI_REQUIRE(ctx, lin->kind == PI_BF16 && a.x_bf16 && a.M >= 1, "the bf16 GEMM takes bf16 weights and activations");
  PI_REQUIRE(ctx, (uintptr_t)a.x_bf16 % 16 == 0 && a.x_stride % 8 == 0 && (uintptr_t)lin->w % 16 == 0 && lin->ld % 8 == 0,
             "bf16 operands must start and step on 16-byte boundaries");
  const pi_expert_rows* ex = a.experts;
  PI_REQUIRE(ctx, !ex || (ex->experts > 0 && lin->rows % ex->experts == 0 && ex->tiles && ex->n_tiles && ex->max_tiles > 0), "a stack of experts needs its tile table");
  const int N = (int)(ex ? lin->rows / ex->experts : lin->rows);
  const bool glu = pi_epi_glu(a.epi) && a.out_bf16 && (a.glu_rows ? a.glu_rows % 2 == 0 && a.glu_rows <= N && a.rest : N % 2 == 0);
  PI_REQUIRE(ctx, a.epi == PI_EPI_STORE || glu || (a.epi == PI_EPI_MAPS_QKV && a.maps_kv && a.maps_kv->dim % 2 == 0) ||
                      (a.epi == PI_EPI_SCALE_ADD && a.out && a.out_scale) || (a.epi == PI_EPI_GELU_TABLE && a.out_bf16 && a.table.base && a.table.tokens) ||
                      (a.epi == PI_EPI_RELU2 && a.out_bf16) ||
                      (a.epi == PI_EPI_DYT_RESIDUAL && a.residual && a.residual->x && a.residual->h && a.residual->post.w && a.residual->next.w),
             "this epilogue is not built for the bf16 GEMM");
  Bf16GemmParams p = {};
  p.out = a.out;
  p.out_bf16 = a.out_bf16;
  p.out_stride = a.out_stride;
  p.out_scale = a.out_scale;
  p.table = a.table;
  p.glu_limit = a.glu_limit;
  p.glu_rows = a.glu_rows ? a.glu_rows : N;
  p.rest = a.rest;
  p.rest_stride = a.rest_stride;
  p.N = N;
  p.K = (int)lin->cols;
  p.M = a.M;
  p.nkb = (p.K + kTK - 1) / kTK;
  p.rtiles = (p.N + kTM - 1) / kTM;
  p.epi = a.epi;
  if (a.residual) p.res = *a.residual;
  if (a.maps_kv) p.mkv = *a.maps_kv;
  p.err_flag = ctx->dev_err;
  int bn = a.M <= 16 ? 16 : a.M <= 32 ? 32 : a.M <= 64 ? 64 : 128;
  if (a.M > 128) {   // the wider tile where it does not cost more rounds of tiles over the SMs
    const long t128 = (long)p.rtiles * ((a.M + 127) / 128), t256 = (long)p.rtiles * ((a.M + 255) / 256), sms = ctx->sm_count;
    if ((t256 + sms - 1) / sms * 3 <= (t128 + sms - 1) / sms * 2) bn = 256;
  }
  if (ex) {
    bn = ex->tile_rows;
    p.tile_table = ex->tiles;
    p.n_tiles = ex->n_tiles;
  }
  p.tiles = p.rtiles * (ex ? ex->max_tiles : (a.M + bn - 1) / bn);
  CUtensorMap w, x;
  PI_TRY(encode_2d(ctx, &w, lin->w, lin->cols, lin->rows, lin->ld, kTM));
  PI_TRY(encode_2d(ctx, &x, a.x_bf16, lin->cols, a.M, a.x_stride, bn));
  pi_prof_scope prof(ctx, PI_PROF_GEMM_TC);
  cudaError_t e;
  if (ex) {
    switch (bn) {
      case 16: e = run_grouped<16, 8>(ctx, p, w, x); break;
      case 32: e = run_grouped<32, 8>(ctx, p, w, x); break;
      case 64: e = run_grouped<64, 6>(ctx, p, w, x); break;
      case 128: e = run_grouped<128, 4>(ctx, p, w, x); break;
      case 256: e = run_grouped<256, 4>(ctx, p, w, x); break;
      default: return pi_fail(ctx, PI_ERR_INVALID_ARG, "expert tiles of %d rows are not built", bn);
    }
  } else switch (bn) {
    case 16: e = run<16, 8>(ctx, p, w, x); break;
    case 32: e = run<32, 8>(ctx, p, w, x); break;
    case 64: e = run<64, 6>(ctx, p, w, x); break;
    case 128: e = run<128, 4>(ctx, p, w, x); break;
    default: e = run<256, 4>(ctx, p, w, x); break;
  }
  if (e != cudaSuccess) return pi_fail(ctx, PI_ERR_CUDA, "bf16 GEMM launch failed: %s", cudaGetErrorString(e));
  ctx->launches++;
  return PI_OK;
}
