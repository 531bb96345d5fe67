// Internal declarations of layered designs: models whose layers each name a token mixer (windowed multi-map attention,
// latent attention, a gated linear recurrence, a matrix memory, a state-space recurrence, lightning attention, minGRU) and a
// feed-forward (dense or experts) with sizes of their own.
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
  // latent attention: rows that attend to the cached latents as they are, and the portions that are long enough to have their
  // keys and values spelled out first.  Those portions see keys from exp_lo[seq] on (a multiple of kExpandBlock); their
  // expanded rows lie in a scratch pool with tables of its own, positions counted from exp_lo.
  const int32_t* latent_rows = nullptr;
  int n_latent = 0;
  const int32_t* expand = nullptr;      // sequences
  int n_expand = 0, max_expand = 0;     // ... their longest portion
  const int32_t* exp_lo = nullptr;      // [n_seqs]
  const int32_t* exp_start = nullptr;   // [n_seqs] position of the portion's first token, from exp_lo
  const int32_t* exp_lens = nullptr;    // [n_seqs]
  const int32_t* exp_tables = nullptr;  // [n_seqs][exp_max_blocks]
  int exp_max_blocks = 0, exp_blocks = 0;
  const int32_t* key_seq = nullptr;     // [n_keys] of every expanded key: sequence, position from exp_lo
  const int32_t* key_pos = nullptr;
  int n_keys = 0;
};
constexpr int kExpandBlock = 64;        // tokens of a block of the expanded pool
constexpr int kExpandPortion = 64;      // a portion of at least this many tokens is expanded

// ---- multi-map attention (pi_attention_maps.cu) -----------------------------------------------------------------
// Per query head `maps` softmax maps over the same values.  maps == 1: plain attention.  maps == 2: the difference
// a1 - lambda a2, brought to unit root mean square over the head and scaled by out_scale.
struct pi_maps_attention {
  int heads = 0, kv_heads = 0, maps = 1, dim = 0, vdim = 0;
  int window = 0;                       // <= 0: everything before
  float scale = 1.f, eps = 0.f;
  float lambda = 0.f, out_scale = 1.f;  // maps == 2
  const float* gate = nullptr;          // the result is multiplied by sigmoid(gate[row][heads * vdim]), or [row][heads]
  size_t gate_stride = 0;
  bool gate_per_head = false;
  const float* slopes = nullptr;        // [heads] taken off a score per token of distance
  const float* sinks = nullptr;         // [heads] exp(sink) joins the sum of weights, once, without a value
  const float* sigmoid_bias = nullptr;  // [heads] a key weighs sigmoid(score + bias) instead, not normalised (maps == 1; no slopes, sinks)
  bool v_in_k = false;                  // the values are the first channels of the keys (f32 kernel)
  int rot_dims = 0;
  const float* rope_cos = nullptr;      // [positions][rot_dims / 2]
  const float* rope_sin = nullptr;
};
struct pi_kv_view {                     // one layer's region of the pool
  void* base = nullptr;
  int kind = PI_F32, kv_heads = 0, maps = 0, dp = 0, vp = 0, block_size = 0;
};
// What happens to q, k and v between projection and attention beside the rotation (all optional; norm_qk stands alone).
struct pi_maps_prepare {
  const float* norm_qk = nullptr;       // [q | k] weights of an RMS norm over all of q, and one over all of k (eps of the attention)
  bool q_only = false;                  // k and v are another layer's
  const float* bias = nullptr;          // [q | k | v]
  bool unit_qk = false;                 // q and k over their root mean square, per head and map (eps of the attention)
  const float* q_temp = nullptr;        // [positions] factor of q
  pi_value_mix mix;
};
// Bring q (in place), k and v of every row into their final form and write k and v into the pool.  qkv rows: [q: heads*maps*dim |
// k | v].
pi_status pi_launch_maps_prepare(pi_ctx* ctx, const pi_maps_attention& a, const pi_maps_prepare& x, const pi_kv_view& kv, float* qkv, size_t stride,
                                 const pi_seq_batch& b);
// out[row][heads * vdim] as f32 or bf16 (out_kind).
pi_status pi_launch_maps_attention(pi_ctx* ctx, const pi_maps_attention& a, const pi_kv_view& kv, const float* qkv, size_t stride,
                                   void* out, size_t out_stride, int out_kind, const pi_seq_batch& b);

// ---- latent attention (pi_latent.cu) ------------------------------------------------------------------------------
// Keys and values of all heads are linear in one latent vector c per token; beside it a rotated key part common to the
// heads.  Only these two are cached: pool rows [c, padded to 16 | rotated part, padded to 16], one kv head, no V part.
struct pi_latent_attention {
  int heads = 0, dim = 0, rot_dims = 0, vdim = 0, rank = 0, window = 0;
  float scale = 1.f, eps = 0.f;
  const float* norm = nullptr;          // [rank]
  const pi_linear* uk_t = nullptr;      // [heads * rank][dim]: a head's unrotated query into latent space
  const pi_linear* ukv = nullptr;       // [heads * dim + heads * vdim][rank]
  const float* rope_cos = nullptr;      // [positions][rot_dims / 2]
  const float* rope_sin = nullptr;
  int col_q = 0, col_kv = 0, col_g = 0; // columns of the fused projection: queries [head][dim | rot], [c | rotated key], gate
};
struct pi_latent_scratch {
  void* q = nullptr;                    // [rows][heads][dp] queries in the layout of a pool row, pool's type
  void* o = nullptr;                    // [rows][heads][rank] weighted latents
  __nv_bfloat16 *keys = nullptr, *pool = nullptr;   // expanded portions: latents of the keys [n_keys][rp], scratch pool
};
inline int pi_latent_rp(int rank) { return (rank + 15) / 16 * 16; }
inline int pi_latent_dp(int rank, int rot) { return pi_latent_rp(rank) + (rot + 15) / 16 * 16; }
bool pi_latent_expandable(const pi_ctx* ctx, const pi_latent_attention& a, int compute);
bool pi_latent_supported(const pi_ctx* ctx, const pi_latent_attention& a, int compute);
size_t pi_latent_pool_elems(const pi_latent_attention& a, int blocks);   // scratch pool of that many blocks
// out[row][heads * vdim], gated, as f32 or bf16 (out_kind).
pi_status pi_launch_latent_attention(pi_ctx* ctx, const pi_latent_attention& a, const pi_kv_view& kv, float* proj, size_t stride, void* out,
                                     size_t out_stride, int out_kind, const pi_seq_batch& b, const pi_latent_scratch& s);

// ---- state-space recurrence (pi_ssd.cu, pi_ssd_chunk.cu) ---------------------------------------------------------------
struct pi_ssd {
  int heads = 0, vdim = 0, dim = 0, groups = 1, norm_groups = 1, taps = 1;   // dim: state channels
  float eps = 0.f;
  const float *conv = nullptr, *conv_b = nullptr;   // [channels][taps], [channels]; channels: x, B, C.  Null: no convolution (taps 1)
  const float4* conv4 = nullptr;        // up to four taps: the same, with zeros in front
  const float *dt_bias = nullptr, *a_log = nullptr, *d = nullptr;   // [heads]
  // a constant decay per head instead: dt = 1, no dt column, dt_bias, a_log and d are null
  const float *decay = nullptr, *log_decay = nullptr;   // [heads]
  bool gate_last = false;               // out = norm(y) sigmoid(z) instead of norm(y silu(z))
  const float* norm = nullptr;          // [heads * vdim]
  int col_z = 0, col_x = 0, col_dt = 0; // columns of the fused projection: z | x, B, C | dt
  // state: per slot S [heads][dim][vdim], then the convolution's last inputs [taps - 1][channels]
  float* state = nullptr;
  size_t state_stride = 0, state_off = 0;
  __host__ __device__ int inner() const { return heads * vdim; }
  __host__ __device__ int channels() const { return heads * vdim + 2 * groups * dim; }
  size_t state_floats() const { return ((size_t)heads * dim * vdim + (size_t)(taps - 1) * channels() + 31) / 32 * 32; }
};
// y: f32 scratch [rows][heads * vdim]; out: the gated, normalised result.
pi_status pi_launch_ssd(pi_ctx* ctx, const pi_ssd& r, const float* proj, size_t stride, float* y, void* out, size_t out_stride, int out_kind,
                        const pi_seq_batch& b, float* scratch);
size_t pi_ssd_scratch_floats(const pi_ssd& r, int n_chunks);
bool pi_ssd_chunked(const pi_ctx* ctx, const pi_ssd& r, int compute);
pi_status pi_launch_ssd_chunks(pi_ctx* ctx, const pi_ssd& r, const float* proj, size_t stride, float* y, const pi_seq_batch& b, float* scratch);

// ---- experts (pi_moe.cu; the products are pi_linear with pi_expert_rows) ---------------------------------------------------
struct pi_moe {
  int experts = 0, top = 0, groups = 1, keep = 1;
  int score = PI_SCORE_SIGMOID, group_best = 2, renorm = 1;
  float scale = 1.f;                    // of the weights
  const float* bias = nullptr;          // [experts], of the logits
  const float* correction = nullptr;    // [experts], part of the choice and not of the weights
};
struct pi_moe_lists {
  int32_t* ids = nullptr;               // [rows][top]
  float* weights = nullptr;             // [rows][top]
  int32_t *place = nullptr, *pair_at = nullptr;   // [rows * top] where a pair lies among the rows grouped by expert, and back
  int4* tiles = nullptr;
  int32_t* n_tiles = nullptr;
};
int pi_moe_tile_rows(int rows, const pi_moe& m);
int pi_moe_max_tiles(int rows, const pi_moe& m);
pi_status pi_launch_moe_route(pi_ctx* ctx, const pi_moe& m, const float* logits, size_t stride, int rows, const pi_moe_lists& l);
pi_status pi_launch_moe_gather(pi_ctx* ctx, const pi_moe& m, int rows, const pi_moe_lists& l, const __nv_bfloat16* h, size_t ld_h, __nv_bfloat16* out);

// ---- rows: residual stream and norms (pi_rows.cu) -------------------------------------------------------------------
struct pi_layer_norm {
  const float* w = nullptr;
  float eps = 0.f;
};
// scale (sum over k of weights[row][k] y[place[row][k]] + sigmoid(shared_gate[row]) shared[row]); null: no gate, no scale
struct pi_expert_sum {
  int top = 0;
  const float* weights = nullptr;
  const int32_t* place = nullptr;       // null: row * top + k
  const void* y = nullptr;
  int y_bf16 = 0;
  size_t y_stride = 0;
  const float *shared = nullptr, *shared_gate = nullptr;
  size_t shared_stride = 0, shared_gate_stride = 0;
  const float* scale = nullptr;         // [width]
};
// A table of token pairs beside the embedding: row (previous token mul_prev + token mul_cur) mod buckets, for a sequence's first token
// row `buckets`.  The previous token of a portion's first row is in the sequence's state slot; the step leaves its last token there.
struct pi_token_pairs {
  const uint16_t* table = nullptr;
  size_t ld = 0;
  int buckets = 0, mul_prev = 0, mul_cur = 0;
  const int32_t *row_seq = nullptr, *seq_row0 = nullptr, *seq_n = nullptr, *seq_start = nullptr, *slot = nullptr;
  float* state = nullptr;               // the token as an integer, in the first word of a slot
  size_t state_stride = 0;
};
struct pi_row_norm {
  bool rms = false;                     // RMS norms (weights as they multiply) instead of layer norm; then also:
  const float* y = nullptr;             //   x += post(y) first; post applies to the experts' sum too
  size_t y_stride = 0;
  pi_layer_norm post;
  bool of_sum = false;                  //   x = post(keep x + y) instead
  float keep = 1.f;
  const float *gate = nullptr, *gate_bias = nullptr;   // the result times sigmoid(gate[row][.] + gate_bias[.]) (null: not)
  size_t gate_stride = 0;
  float embed_scale = 1.f;              //   x = embed_scale table[token] + pairs[its pair]
  pi_token_pairs pairs;
                                        //   norm.w null: h is x as it stands
  int rows = 0, width = 0;
  float* x = nullptr;                   // [.][width]
  const int32_t* pick = nullptr;        // row i is x[pick[i]]
  const uint16_t* table = nullptr;      // x = table[token] first (the first kernel of a step)
  size_t table_ld = 0;
  int vocab = 0;
  const uint32_t* tokens = nullptr;
  const pi_expert_sum* experts = nullptr;   // x += experts first
  pi_layer_norm norm;
  void* h = nullptr;                    // null: no normalised row is wanted
  size_t ld_h = 0;
  int h_kind = PI_F32;
};
pi_status pi_launch_row_norm(pi_ctx* ctx, const pi_row_norm& n);

// ---- the token table beside the layers (pi_side.cu) ---------------------------------------------------------------------------
struct pi_token_side {
  const pi_linear *gate = nullptr, *proj = nullptr;   // [dim][width], [width][dim]
  pi_token_table table;                 // the layer's columns
  pi_layer_norm post;                   // RMS norm of what it adds
};
constexpr int kSideRows = 8;            // steps of up to this many rows
bool pi_token_side_usable(const pi_ctx* ctx, const pi_token_side& s, int rows, int width);
// What the sublayer before left (n.y or n.experts, with n.post), the token's contribution, and n.h.
pi_status pi_launch_token_side(pi_ctx* ctx, const pi_token_side& s, const pi_row_norm& n);

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

// ---- minGRU (pi_mingru.cu) -------------------------------------------------------------------------------------------
// S = (1 - z) S + z c per channel, z = sigmoid(zl), c = u + 1/2 (u >= 0) or sigmoid(u); out = S silu(g).
struct pi_mingru {
  int width = 0;
  const float *z_bias = nullptr, *x_bias = nullptr;   // [width]
  int col_z = 0, col_x = 0, col_g = 0;  // columns of the fused projection
  float* state = nullptr;               // S [width] per slot
  size_t state_stride = 0, state_off = 0;
  size_t state_floats() const { return ((size_t)width + 31) / 32 * 32; }
};
pi_status pi_launch_mingru(pi_ctx* ctx, const pi_mingru& r, const float* proj, size_t stride, void* out, size_t out_stride, int out_kind,
                           const pi_seq_batch& b);

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
