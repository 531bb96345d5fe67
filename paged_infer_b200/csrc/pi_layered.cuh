// Internal declarations of layered designs: models whose layers each name a token mixer (windowed multi-map attention,
// a gated linear recurrence, a matrix memory) with sizes of its own.
#pragma once

#include "pi_common.cuh"

// ---- one ragged step ------------------------------------------------------------------------------------------
// n_seqs sequences bring seq_n[i] >= 1 consecutive tokens each; their rows lie one after the other.  All pointers are
// device memory; everything here was uploaded before the step's first kernel (the embedding, which waits strictly), so
// kernels may read it ahead of their own dependency wait.
struct pi_seq_batch {
  int n_seqs = 0, rows = 0;
  const uint32_t* tokens = nullptr;     // [rows]
  const int32_t* row_seq = nullptr;     // [rows]
  const int32_t* row_pos = nullptr;     // [rows]
  const int32_t* seq_row0 = nullptr;    // [n_seqs]
  const int32_t* seq_n = nullptr;       // [n_seqs]
  const int32_t* seq_start = nullptr;   // [n_seqs] position of the first token of the portion
  const int32_t* slot = nullptr;        // [n_seqs] state slot
  const int32_t* lens = nullptr;        // [n_seqs] mapped blocks
  const int32_t* tables = nullptr;      // [n_seqs][max_blocks]
  int max_blocks = 0;
  // attention work: rows that are decoded alone, and (sequence, first row in it) of the query tiles of longer portions
  const int32_t* single_rows = nullptr;
  int n_single = 0;
  const int32_t* portions = nullptr;    // sequences that bring several tokens
  int n_portions = 0;
  int max_portion = 0;                  // longest of them
  // recurrence work: sequences for the token-by-token kernel, and those long enough for the chunked one
  const int32_t* scan_seqs = nullptr;
  int n_scan = 0;
  const int32_t* chunk_seqs = nullptr;
  int n_chunk_seqs = 0;
  const int32_t* chunks = nullptr;      // [n_chunks][2]: index into chunk_seqs, first token of the chunk
  int n_chunks = 0;
  const int32_t* chunk0 = nullptr;      // [n_chunk_seqs + 1] first chunk of a sequence
  int max_pos = 0;                      // host-side bound on every position of the step
};

// ---- multi-map attention (pi_attention_maps.cu) -----------------------------------------------------------------
// Per query head `maps` softmax maps over the same values.  maps == 1: plain attention.  maps == 2: the difference
// a1 - lambda a2, brought to unit root mean square over the head and scaled by out_scale.
struct pi_maps_attention {
  int heads = 0, kv_heads = 0, maps = 1, dim = 0, vdim = 0;
  int window = 0;                       // <= 0: everything before
  float scale = 1.f, eps = 0.f;
  float lambda = 0.f, out_scale = 1.f;  // maps == 2
  int rot_dims = 0;
  const float* rope_cos = nullptr;      // [positions][rot_dims / 2]
  const float* rope_sin = nullptr;
};
struct pi_kv_view {                     // one layer's region of the pool
  void* base = nullptr;
  int kind = PI_F32, kv_heads = 0, maps = 0, dp = 0, vp = 0, block_size = 0;
};
// Rotate q (in place) and k, and write k and v of every row into the pool.  qkv rows: [q: heads*maps*dim | k | v].
pi_status pi_launch_maps_rope_kv(pi_ctx* ctx, const pi_maps_attention& a, const pi_kv_view& kv, float* qkv, size_t stride,
                                 const pi_seq_batch& b);
// out[row][heads * vdim] as f32 or bf16 (out_kind).
pi_status pi_launch_maps_attention(pi_ctx* ctx, const pi_maps_attention& a, const pi_kv_view& kv, const float* qkv, size_t stride,
                                   void* out, size_t out_stride, int out_kind, const pi_seq_batch& b);

// ---- recurrences (pi_recurrent.cu) --------------------------------------------------------------------------------
enum pi_recurrence_kind { PI_REC_GLA = 0, PI_REC_MLSTM = 1 };
struct pi_recurrence {
  int kind = PI_REC_GLA;
  int heads = 0, dim = 0, vdim = 0;
  float eps = 0.f;
  float q_scale = 1.f;
  const float* norm = nullptr;          // [vdim] shared by the heads, or [heads * vdim]
  bool norm_per_head = false;
  int gate_sigmoid = 0;                 // output gate: 0 silu, 1 sigmoid
  // GLA: log decay = log_sigmoid(a2 (low-rank input) + a2_b) / tau per key channel
  float tau = 1.f;
  int rank = 0;
  const float* a2 = nullptr;            // [heads * dim][rank]
  const float* a2_b = nullptr;
  // mLSTM: log gates cap tanh((x + bias) / cap), the forget one behind a log_sigmoid
  float gate_cap = 1.f;
  const float *i_b = nullptr, *f_b = nullptr;   // [heads]
  // columns of the fused projection
  int col_q = 0, col_k = 0, col_v = 0, col_g = 0, col_low = 0, col_i = 0, col_f = 0;
  // state: per slot, `state_stride` floats, this layer's part at state_off: S [heads][dim][vdim], then for the mLSTM
  // n [heads][dim] and m [heads]
  float* state = nullptr;
  size_t state_stride = 0, state_off = 0;
};
inline size_t pi_recurrence_floats(int kind, int heads, int dim, int vdim) {
  const size_t s = (size_t)heads * dim * vdim + (kind == PI_REC_MLSTM ? (size_t)heads * (dim + 1) : 0);
  return (s + 31) / 32 * 32;
}
// out[row][heads * vdim]: normalised, gated head outputs as f32 or bf16.  `scratch`: see pi_recurrence_scratch_floats.
pi_status pi_launch_recurrence(pi_ctx* ctx, const pi_recurrence& r, const float* proj, size_t stride, void* out, size_t out_stride,
                               int out_kind, const pi_seq_batch& b, float* scratch);
size_t pi_recurrence_scratch_floats(const pi_recurrence& r, int n_chunks);
// The chunked kernels (pi_recurrent_chunk.cu) for the sequences of b.chunk_seqs.
pi_status pi_launch_recurrence_chunks(pi_ctx* ctx, const pi_recurrence& r, const float* proj, size_t stride, __nv_bfloat16* out, size_t out_stride,
                                      const pi_seq_batch& b, float* scratch);
// A portion of at least this many tokens takes the chunked kernels (when they hold the layer's sizes).
constexpr int kRecurrenceChunk = 64;
bool pi_recurrence_chunked(const pi_ctx* ctx, const pi_recurrence& r, int compute);

// ---- row-wise glue (pi_layered.cu) -----------------------------------------------------------------------------------
template <typename K, typename... Args>
inline cudaError_t pi_launch_dep(pi_ctx* ctx, K k, dim3 grid, dim3 block, size_t smem, int cluster_x, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = ctx->stream;
  cudaLaunchAttribute attr[2];
  int na = 0;
  if (ctx->opt_pdl) {
    attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[na].val.programmaticStreamSerializationAllowed = 1;
    ++na;
  }
  if (cluster_x > 1) {
    attr[na].id = cudaLaunchAttributeClusterDimension;
    attr[na].val.clusterDim.x = cluster_x;
    attr[na].val.clusterDim.y = 1;
    attr[na].val.clusterDim.z = 1;
    ++na;
  }
  cfg.attrs = attr;
  cfg.numAttrs = na;
  return cudaLaunchKernelEx(&cfg, k, args...);
}
#define PI_LAUNCH_OK(ctx, e)                                                                            \
  do {                                                                                                  \
    cudaError_t _le = (e);                                                                              \
    if (_le != cudaSuccess)                                                                             \
      return pi_fail((ctx), PI_ERR_CUDA, "kernel launch failed: %s (%s:%d)", cudaGetErrorString(_le),  \
                     __FILE__, __LINE__);                                                               \
    (ctx)->launches++;                                                                                  \
  } while (0)

#ifdef __CUDACC__
template <typename T>
__device__ __forceinline__ T pi_from_f32(float v);
template <>
__device__ __forceinline__ float pi_from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 pi_from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float pi_to_f32(float v) { return v; }
__device__ __forceinline__ float pi_to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
#endif

// ---- the model (pi_layered.cu) -------------------------------------------------------------------------------------
// The layered model behind a handle, or null: then *L is the uniform layout (without block count and size).
const pi_layered* pi_model_layered(const pi_model* model, pi_kv_layout* L);
pi_status pi_layered_create(pi_ctx* ctx, const pi_layered_config* cfg, const pi_named_tensor* tensors, int n_tensors, int gla_rank,
                            uint64_t seed, float std, pi_layered** out);   // tensors == nullptr: synthetic
void pi_layered_destroy(pi_layered* m);
size_t pi_layered_weight_bytes(const pi_layered* m);
int pi_layered_max_rows(const pi_layered* m);
int pi_layered_vocab(const pi_layered* m);
size_t pi_layered_state_floats(const pi_layered* m);
pi_status pi_layered_kv_regions(pi_ctx* ctx, const pi_layered* m, int num_blocks, int block_size, pi_kv_pool* pool);
pi_status pi_layered_step(pi_ctx* ctx, pi_layered* m, pi_kv_pool* pool, pi_state_pool* state, const pi_step_batch* batch,
                          float* logits_host, uint32_t* argmax_host);
pi_status pi_layered_step_multi(pi_ctx* ctx, pi_layered* m, pi_kv_pool* pool, pi_state_pool* state, const pi_step_batch* batch, int n_steps,
                                uint32_t* out_tokens_host);
pi_status pi_layered_trace(pi_ctx* ctx, pi_layered* m, int on);
pi_status pi_layered_read_layer(pi_ctx* ctx, const pi_layered* m, int layer, int rows, float* out);
