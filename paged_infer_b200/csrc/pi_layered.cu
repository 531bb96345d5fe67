// Layered designs: a decoder whose layers each name a token mixer - windowed attention with one or two softmax maps, a
// gated linear recurrence (GLA), a matrix memory (mLSTM) - and, if they have one, a gelu-gated feed-forward; every
// sublayer normalised before and after by Dynamic Tanh, embedding tied to the output.
//
//   x += dyt(norm1b, mixer(dyt(norm1, x)));   x += dyt(norm2b, ff(dyt(norm2, x)))
//
// Dynamic Tanh needs no statistics, so all of it folds into the projection that ends a sublayer: its epilogue adds
// the normalised result to the f32 residual stream and hands on the normalised input of the next sublayer.  Per layer:
//   1. [q;k;v(;gates)] projection; attention: rotary positions and the KV write in its epilogue
//   2. attention (with its own normalisation in the same kernel); or the recurrence with head norm and output gate in the
//      same kernel
//   3. output projection, epilogue = residual update + next norm
//   4. interleaved [gate;up] projection, epilogue = gelu(gate) * up      (layers with a feed-forward)
//   5. down projection, epilogue = residual update + next norm
// In the bf16 mode projections of more than opt_gemv_max_m rows run on tcgen05 with bf16 activations, smaller ones on
// the CUDA cores with f32 activations; the f32 mode keeps f32 activations, KV and CUDA-core arithmetic throughout (the
// bf16 weights widen exactly).  The residual stream, recurrent state, scores and gates are f32 in both.
#include <math.h>
#include <string.h>

#include <algorithm>
#include <map>
#include <new>
#include <string>

#include "pi_layered.cuh"
#include "pi_load.cuh"

using pi_load::build_linear;
using pi_load::Piece;
using pi_load::Source;

struct pi_state_pool {
  float* data = nullptr;
  size_t stride = 0;     // floats per slot
  int slots = 0;
};

namespace {

struct Layer {
  pi_layer_config c;
  pi_dyt norm1, norm1b, norm2, norm2b;
  pi_linear *in = nullptr, *out = nullptr, *gate_up = nullptr, *down = nullptr;
  int attn = -1;                 // index of the layer's KV region
  int rope = -1;                 // index of its rotary table
  float lambda = 0.f;
  pi_recurrence rec;
};

struct RopeTable {
  int dims = 0, cap = 0;
  float base = 1.f;
  float *cos = nullptr, *sin = nullptr;
};

}  // namespace

struct pi_layered {
  pi_layered_config c;
  std::vector<Layer> layers;
  std::vector<RopeTable> ropes;
  std::vector<void*> owned;      // device vectors
  pi_linear* embed = nullptr;
  pi_dyt final_norm;
  size_t weight_bytes = 0, state_floats = 0;
  bool chunked = false;          // every recurrent layer has a chunked kernel
  // scratch for c.max_rows rows; activations are sized for f32 and hold bf16 on the tensor path
  float *x = nullptr, *proj = nullptr;
  void *h = nullptr, *core = nullptr, *ffh = nullptr;
  size_t ld_h = 0, ld_core = 0, ld_ff = 0, ld_proj = 0;
  pi_buffer meta, head_in, logits, ids, scratch, trace, history;
  bool trace_on = false;
  cudaGraphExec_t step_exec = nullptr;
};

namespace {

size_t round8(size_t n) { return (n + 7) / 8 * 8; }

template <typename T>
__device__ __forceinline__ void store_act(void* p, size_t i, float v) { static_cast<T*>(p)[i] = pi_from_f32<T>(v); }

// x = embed[token], h = dyt(norm, x).  Strict wait: see pi_seq_batch.
template <typename T>
__global__ void __launch_bounds__(256) embed_dyt_kernel(const uint16_t* __restrict__ table, size_t ld, int vocab, int width,
                                                        const uint32_t* __restrict__ tokens, float* __restrict__ x, pi_dyt norm, void* h,
                                                        size_t ld_h) {
  pi_grid_dependency_wait_strict();
  const int row = blockIdx.x;
  const uint16_t* src = table + (size_t)(tokens[row] % (uint32_t)vocab) * ld;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float v = pi_bf16_bits_to_f32(src[i]);
    x[(size_t)row * width + i] = v;
    store_act<T>(h, (size_t)row * ld_h + i, pi_dyt_apply(norm, v, i));
  }
}

// h[i] = dyt(norm, x[rows[i]])
template <typename T>
__global__ void __launch_bounds__(256) gather_dyt_kernel(const float* __restrict__ x, int width, const int32_t* __restrict__ rows,
                                                         pi_dyt norm, void* h, size_t ld_h) {
  const int row = rows[blockIdx.x];
  pi_grid_dependency_wait();
  for (int i = threadIdx.x; i < width; i += blockDim.x)
    store_act<T>(h, (size_t)blockIdx.x * ld_h + i, pi_dyt_apply(norm, x[(size_t)row * width + i], i));
}

// After a greedy step of single tokens: the chosen ids become the next tokens, every sequence moves on one position.
__global__ void advance_seqs_kernel(uint32_t* tokens, const uint32_t* chosen, uint32_t* history, int* counter, int32_t* row_pos,
                                    int32_t* seq_start, int n) {
  pi_grid_dependency_wait();
  const int step = *counter;
  for (int b = threadIdx.x; b < n; b += blockDim.x) {
    tokens[b] = chosen[b];
    history[(size_t)step * n + b] = chosen[b];
    row_pos[b] += 1;
    seq_start[b] += 1;
  }
  __syncthreads();
  if (threadIdx.x == 0) *counter = step + 1;
}

// ---- weights ----------------------------------------------------------------------------------------------------------
struct Loader {
  pi_ctx* ctx;
  pi_layered* m;
  std::map<std::string, const pi_named_tensor*> by_name;
  std::vector<pi_tensor> keep;     // stable storage for Source::host
  bool synthetic = false;
  uint64_t seed = 0, next_stream = 1;
  float std = 0.02f;

  pi_status find(const std::string& name, const pi_named_tensor** out) {
    auto it = by_name.find(name);
    PI_REQUIRE(ctx, it != by_name.end(), "missing tensor: %s", name.c_str());
    *out = it->second;
    return PI_OK;
  }
  pi_status vec(const std::string& name, size_t n, std::vector<float>* out, float fill = 0.f) {
    if (synthetic) {
      out->assign(n, fill);
      return PI_OK;
    }
    const pi_named_tensor* t;
    PI_TRY(find(name, &t));
    PI_REQUIRE(ctx, (size_t)(t->rows * t->cols) == n, "%s has %lld elements, the configuration says %zu", name.c_str(),
               (long long)(t->rows * t->cols), n);
    out->resize(n);
    for (size_t i = 0; i < n; ++i) {
      if (t->kind == PI_F32) {
        (*out)[i] = static_cast<const float*>(t->data)[i];
      } else {
        const uint32_t u = (uint32_t)static_cast<const uint16_t*>(t->data)[i] << 16;
        memcpy(&(*out)[i], &u, 4);
      }
    }
    return PI_OK;
  }
  pi_status dev_vec(const std::string& name, size_t n, const float** out, float fill = 0.f) {
    std::vector<float> v;
    PI_TRY(vec(name, n, &v, fill));
    float* d = nullptr;
    PI_CUDA(ctx, cudaMalloc(&d, std::max<size_t>(n, 1) * sizeof(float)));
    m->owned.push_back(d);
    PI_CUDA(ctx, cudaMemcpy(d, v.data(), n * sizeof(float), cudaMemcpyHostToDevice));
    *out = d;
    return PI_OK;
  }
  pi_status dyt(const std::string& name, pi_dyt* out) {
    const size_t n = m->c.width;
    std::vector<float> alpha;
    PI_TRY(vec(name + ".alpha", 1, &alpha, 0.5f));
    out->alpha = alpha[0];
    PI_TRY(dev_vec(name, n, &out->w, 1.f));
    return dev_vec(name + ".b", n, &out->b);
  }
  // A matrix of the checkpoint as rows dst_r0, dst_r0 + step, ... of a fused one.
  pi_status piece(const std::string& name, size_t rows, size_t cols, size_t dst_r0, size_t step, std::vector<Piece>* out) {
    Source s;
    s.rows = rows;
    s.cols = cols;
    if (synthetic) {
      s.synthetic = true;
      s.seed = seed;
      s.stream_id = next_stream++;
      s.std = std;
      s.kind = PI_BF16;
    } else {
      const pi_named_tensor* t;
      PI_TRY(find(name, &t));
      PI_REQUIRE(ctx, t->rows == (int64_t)rows && t->cols == (int64_t)cols, "%s is %lld x %lld, the configuration says %zu x %zu",
                 name.c_str(), (long long)t->rows, (long long)t->cols, rows, cols);
      PI_REQUIRE(ctx, t->kind == PI_BF16, "%s: matrices are stored as bf16", name.c_str());
      keep.push_back(pi_tensor{PI_BF16, 0, t->rows, t->cols, t->data, nullptr});
      s.host = &keep.back();
    }
    out->push_back(Piece{s, 0, rows, dst_r0, step});
    return PI_OK;
  }
  pi_status matrix(const std::vector<Piece>& pieces, size_t rows, size_t cols, pi_linear** out) {
    PI_TRY(build_linear(ctx, pieces, rows, cols, 0, out));
    m->weight_bytes += pi_linear_weight_bytes(*out);
    return PI_OK;
  }
};

pi_status check_layer(pi_ctx* ctx, int i, const pi_layer_config& c) {
  PI_REQUIRE(ctx, c.mixer >= PI_MIXER_ATTENTION && c.mixer <= PI_MIXER_MLSTM, "layer %d: unknown mixer %d", i, c.mixer);
  PI_REQUIRE(ctx, c.heads > 0 && c.dim > 0 && c.vdim > 0 && c.ff >= 0, "layer %d: sizes must be positive", i);
  if (c.mixer == PI_MIXER_ATTENTION) {
    PI_REQUIRE(ctx, c.kv_heads > 0 && c.heads % c.kv_heads == 0, "layer %d: %d heads do not share %d key/value heads", i, c.heads, c.kv_heads);
    PI_REQUIRE(ctx, c.maps == 1 || c.maps == 2, "layer %d: %d softmax maps", i, c.maps);
    PI_REQUIRE(ctx, c.rot_dims >= 0 && c.rot_dims % 2 == 0 && c.rot_dims <= c.dim, "layer %d: %d rotary channels of %d", i, c.rot_dims, c.dim);
    PI_REQUIRE(ctx, c.rot_dims == 0 || c.rot_base > 0.f, "layer %d: rotary base must be positive", i);
  } else if (c.mixer == PI_MIXER_GLA) {
    PI_REQUIRE(ctx, c.tau != 0.f, "layer %d: tau is zero", i);
  } else {
    PI_REQUIRE(ctx, c.gate_cap > 0.f, "layer %d: gate_cap must be positive", i);
  }
  return PI_OK;
}

pi_status build(pi_ctx* ctx, const pi_layered_config* cfg, Loader& ld, int gla_rank, pi_layered* m) {
  m->c = *cfg;
  m->c.layers = nullptr;
  const size_t W = cfg->width;
  ld.keep.reserve((size_t)cfg->num_layers * 16 + 4);   // Source::host points into it
  size_t max_in = 0, max_core = 1, max_ff = 1;
  int n_attn = 0;
  bool chunk = true;
  {
    std::vector<Piece> p;
    PI_TRY(ld.piece("embed", cfg->vocab_size, W, 0, 1, &p));
    PI_TRY(ld.matrix(p, cfg->vocab_size, W, &m->embed));
  }
  PI_TRY(ld.dyt("final.norm", &m->final_norm));
  m->layers.resize(cfg->num_layers);
  for (int i = 0; i < cfg->num_layers; ++i) {
    Layer& L = m->layers[i];
    L.c = cfg->layers[i];
    const pi_layer_config& c = L.c;
    PI_TRY(check_layer(ctx, i, c));
    const std::string l = "l" + std::to_string(i), mix = l + ".mix.";
    const size_t core = (size_t)c.heads * c.vdim;
    PI_TRY(ld.dyt(l + ".norm1", &L.norm1));
    PI_TRY(ld.dyt(l + ".norm1b", &L.norm1b));
    std::vector<Piece> p;
    size_t rows = 0;
    auto add = [&](const char* name, size_t n) -> pi_status {
      PI_TRY(ld.piece(mix + name, n, W, rows, 1, &p));
      rows += n;
      return PI_OK;
    };
    if (c.mixer == PI_MIXER_ATTENTION) {
      PI_TRY(add("q", (size_t)c.heads * c.maps * c.dim));
      PI_TRY(add("k", (size_t)c.kv_heads * c.maps * c.dim));
      PI_TRY(add("v", (size_t)c.kv_heads * c.vdim));
      L.attn = n_attn++;
      if (c.maps == 2) {   // lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff, one number for the layer
        double e[2];
        for (int j = 0; j < 2; ++j) {
          std::vector<float> a, b;
          PI_TRY(ld.vec(mix + "lq" + std::to_string(j + 1), c.dim, &a));
          PI_TRY(ld.vec(mix + "lk" + std::to_string(j + 1), c.dim, &b));
          double d = 0;
          for (int k = 0; k < c.dim; ++k) d += (double)a[k] * b[k];
          e[j] = exp(d);
        }
        L.lambda = (float)(e[0] - e[1] + (double)c.diff);
      }
      for (size_t t = 0; t < m->ropes.size() && L.rope < 0; ++t)
        if (m->ropes[t].dims == c.rot_dims && m->ropes[t].base == c.rot_base) L.rope = (int)t;
      if (L.rope < 0) {
        RopeTable t;
        t.dims = c.rot_dims;
        t.base = c.rot_base;
        L.rope = (int)m->ropes.size();
        m->ropes.push_back(t);
      }
    } else {
      pi_recurrence& r = L.rec;
      const size_t hd = (size_t)c.heads * c.dim;
      r.kind = c.mixer == PI_MIXER_GLA ? PI_REC_GLA : PI_REC_MLSTM;
      r.heads = c.heads;
      r.dim = c.dim;
      r.vdim = c.vdim;
      r.eps = cfg->norm_eps;
      r.q_scale = (float)(1.0 / sqrt((double)c.dim));
      r.col_q = 0;
      r.col_k = (int)hd;
      r.col_v = (int)(2 * hd);
      r.col_g = (int)(2 * hd + core);
      PI_TRY(add("q", hd));
      PI_TRY(add("k", hd));
      PI_TRY(add("v", core));
      PI_TRY(add("g", core));
      if (r.kind == PI_REC_GLA) {
        r.tau = c.tau;
        r.rank = gla_rank;
        if (!ld.synthetic) {   // the rank is what the checkpoint's matrix has
          const pi_named_tensor* t;
          PI_TRY(ld.find(mix + "a1", &t));
          r.rank = (int)t->rows;
        }
        r.col_low = (int)rows;
        PI_TRY(add("a1", r.rank));
        std::vector<float> a2;
        PI_TRY(ld.dev_vec(mix + "a2", hd * r.rank, &r.a2, 0.01f));
        PI_TRY(ld.dev_vec(mix + "a2.b", hd, &r.a2_b, 2.f));
        PI_TRY(ld.dev_vec(mix + "norm", c.vdim, &r.norm, 1.f));
      } else {
        r.gate_cap = c.gate_cap;
        r.gate_sigmoid = 1;
        r.norm_per_head = true;
        r.col_i = (int)rows;
        PI_TRY(add("i", c.heads));
        r.col_f = (int)rows;
        PI_TRY(add("f", c.heads));
        PI_TRY(ld.dev_vec(mix + "i.b", c.heads, &r.i_b, 0.f));
        PI_TRY(ld.dev_vec(mix + "f.b", c.heads, &r.f_b, 3.f));
        PI_TRY(ld.dev_vec(mix + "norm", core, &r.norm, 1.f));
      }
      r.state_off = m->state_floats;
      m->state_floats += pi_recurrence_floats(r.kind, c.heads, c.dim, c.vdim);
      chunk = chunk && pi_recurrence_chunked(ctx, r, cfg->compute);
    }
    PI_TRY(ld.matrix(p, rows, W, &L.in));
    max_in = std::max(max_in, rows);
    max_core = std::max(max_core, core);
    p.clear();
    PI_TRY(ld.piece(mix + "o", W, core, 0, 1, &p));
    PI_TRY(ld.matrix(p, W, core, &L.out));
    if (c.ff > 0) {
      PI_TRY(ld.dyt(l + ".norm2", &L.norm2));
      PI_TRY(ld.dyt(l + ".norm2b", &L.norm2b));
      p.clear();
      PI_TRY(ld.piece(l + ".mlp.gate", c.ff, W, 0, 2, &p));
      PI_TRY(ld.piece(l + ".mlp.up", c.ff, W, 1, 2, &p));
      PI_TRY(ld.matrix(p, 2 * (size_t)c.ff, W, &L.gate_up));
      p.clear();
      PI_TRY(ld.piece(l + ".mlp.down", W, c.ff, 0, 1, &p));
      PI_TRY(ld.matrix(p, W, c.ff, &L.down));
      max_ff = std::max(max_ff, (size_t)c.ff);
    }
  }
  m->chunked = chunk && m->state_floats > 0;
  const size_t cap = cfg->max_rows;
  m->ld_h = round8(W);
  m->ld_core = round8(max_core);
  m->ld_ff = round8(max_ff);
  m->ld_proj = round8(max_in);
  PI_CUDA(ctx, cudaMalloc(&m->x, cap * W * sizeof(float)));
  PI_CUDA(ctx, cudaMalloc(&m->proj, cap * m->ld_proj * sizeof(float)));
  PI_CUDA(ctx, cudaMalloc(&m->h, cap * m->ld_h * sizeof(float)));
  PI_CUDA(ctx, cudaMalloc(&m->core, cap * m->ld_core * sizeof(float)));
  PI_CUDA(ctx, cudaMalloc(&m->ffh, cap * m->ld_ff * sizeof(float)));
  PI_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  return PI_OK;
}

pi_status ensure_ropes(pi_ctx* ctx, pi_layered* m, int positions) {
  for (RopeTable& t : m->ropes) {
    if (t.dims == 0 || positions <= t.cap) continue;
    const int cap = std::max(positions, std::max(2 * t.cap, 2048)), half = t.dims / 2;
    std::vector<float> c((size_t)cap * half), s(c.size());
    for (int j = 0; j < half; ++j) {
      const double f = pow((double)t.base, -2.0 * j / t.dims);
      for (int p = 0; p < cap; ++p) {
        c[(size_t)p * half + j] = (float)cos(p * f);
        s[(size_t)p * half + j] = (float)sin(p * f);
      }
    }
    PI_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    cudaFree(t.cos);
    cudaFree(t.sin);
    t.cos = t.sin = nullptr;
    PI_CUDA(ctx, cudaMalloc(&t.cos, c.size() * sizeof(float)));
    PI_CUDA(ctx, cudaMalloc(&t.sin, s.size() * sizeof(float)));
    PI_CUDA(ctx, cudaMemcpy(t.cos, c.data(), c.size() * sizeof(float), cudaMemcpyHostToDevice));
    PI_CUDA(ctx, cudaMemcpy(t.sin, s.data(), s.size() * sizeof(float), cudaMemcpyHostToDevice));
    t.cap = cap;
  }
  return PI_OK;
}

// ---- one step -----------------------------------------------------------------------------------------------------------
struct Staged {
  pi_seq_batch b;
  const int32_t* out_rows = nullptr;   // device
  int n_out = 0;
  bool all_rows = false;               // every row, in order
};

// True when a projection over M rows takes bf16 activations (the tensor-core path).
bool act_bf16(const pi_ctx* ctx, const pi_layered* m, int M) {
  return m->c.compute == PI_BF16 && ctx->opt_tensor_gemm && M > ctx->opt_gemv_max_m;
}

pi_status stage(pi_ctx* ctx, pi_layered* m, const pi_kv_pool* pool, const pi_state_pool* state, const pi_step_batch* in, int extra_positions,
                Staged* st) {
  PI_REQUIRE(ctx, in->n_seqs > 0 && in->tokens && in->n_tokens && in->start_pos && in->table_lens, "a step needs at least one sequence");
  PI_REQUIRE(ctx, in->block_tables || in->max_blocks == 0, "null block tables");
  PI_REQUIRE(ctx, m->state_floats == 0 || (state && in->state_slots), "this model carries recurrent state: the step needs a state pool and slots");
  PI_REQUIRE(ctx, m->state_floats == 0 || state->stride == m->state_floats, "the state pool was made for another model");
  PI_REQUIRE(ctx, pool && pool->regions.size() == (size_t)std::count_if(m->layers.begin(), m->layers.end(), [](const Layer& l) { return l.attn >= 0; }) &&
                      pool->kind == m->c.compute,
             "the KV pool was made for another model");
  const int n = in->n_seqs;
  int rows = 0, max_pos = 0;
  std::vector<int32_t> row_seq, row_pos, row0(n), single, portions, scan, chunk_seqs, chunks, chunk0(1, 0);
  int max_portion = 0;
  for (int i = 0; i < n; ++i) {
    const int k = in->n_tokens[i], p0 = in->start_pos[i];
    PI_REQUIRE(ctx, k >= 1 && p0 >= 0 && p0 < (1 << 30), "sequence %d: %d tokens from position %d", i, k, p0);
    PI_REQUIRE(ctx, k <= m->c.max_rows - rows, "the step's tokens exceed the model's %d rows", m->c.max_rows);
    row0[i] = rows;
    for (int j = 0; j < k; ++j) {
      row_seq.push_back(i);
      row_pos.push_back(p0 + j);
    }
    if (k == 1) {
      single.push_back(rows);
    } else {
      portions.push_back(i);
      max_portion = std::max(max_portion, k);
    }
    if (m->chunked && k >= kRecurrenceChunk && act_bf16(ctx, m, k)) {
      for (int t = 0; t < k; t += kRecurrenceChunk) {
        chunks.push_back((int)chunk_seqs.size());
        chunks.push_back(t);
      }
      chunk_seqs.push_back(i);
      chunk0.push_back((int)chunks.size() / 2);
    } else {
      scan.push_back(i);
    }
    rows += k;
    max_pos = std::max(max_pos, p0 + k - 1);
    PI_REQUIRE(ctx, in->table_lens[i] >= 0 && in->table_lens[i] <= in->max_blocks, "sequence %d: %d mapped blocks, tables of %d", i,
               in->table_lens[i], in->max_blocks);
    for (int j = 0; j < in->table_lens[i]; ++j) {
      const int32_t pb = in->block_tables[(size_t)i * in->max_blocks + j];
      PI_REQUIRE(ctx, pb >= 0 && pb < pool->L.num_blocks, "sequence %d maps a block to physical id %d of %d", i, pb, pool->L.num_blocks);
    }
    if (m->state_floats) {
      const int s = in->state_slots[i];
      PI_REQUIRE(ctx, s >= 0 && s < state->slots, "sequence %d: state slot %d of %d", i, s, state->slots);
      for (int j = 0; j < i; ++j) PI_REQUIRE(ctx, in->state_slots[j] != s, "sequences %d and %d share state slot %d", j, i, s);
    }
  }
  PI_REQUIRE(ctx, in->n_out >= 0 && (in->n_out == 0 || in->out_rows), "null output rows");
  st->all_rows = in->n_out == rows;
  for (int i = 0; i < in->n_out; ++i) {
    PI_REQUIRE(ctx, in->out_rows[i] >= 0 && in->out_rows[i] < rows, "output row %d of %d", in->out_rows[i], rows);
    if (in->out_rows[i] != i) st->all_rows = false;
  }
  PI_TRY(ensure_ropes(ctx, m, max_pos + 1 + extra_positions));

  size_t words = 0;
  std::vector<std::pair<const void*, size_t>> parts;
  auto put = [&](const void* src, size_t count) {   // every part starts on a 16-byte boundary
    const size_t at = words;
    parts.push_back({src, count});
    words += (count + 3) / 4 * 4;
    return at;
  };
  const size_t o_tok = put(in->tokens, rows), o_rs = put(row_seq.data(), rows), o_rp = put(row_pos.data(), rows), o_r0 = put(row0.data(), n),
               o_n = put(in->n_tokens, n), o_st = put(in->start_pos, n), o_sl = put(in->state_slots, in->state_slots ? n : 0),
               o_ln = put(in->table_lens, n), o_tb = put(in->block_tables, (size_t)n * in->max_blocks), o_si = put(single.data(), single.size()),
               o_po = put(portions.data(), portions.size()), o_sc = put(scan.data(), scan.size()), o_cs = put(chunk_seqs.data(), chunk_seqs.size()),
               o_ch = put(chunks.data(), chunks.size()), o_c0 = put(chunk0.data(), chunk0.size()), o_out = put(in->out_rows, in->n_out);
  PI_TRY(pi_reserve_pinned(ctx, words * 4));
  PI_TRY(pi_reserve(ctx, &m->meta, words * 4));
  int32_t* host = static_cast<int32_t*>(ctx->pinned);
  size_t at = 0;
  for (auto& q : parts) {
    if (q.second) memcpy(host + at, q.first, q.second * 4);
    at += (q.second + 3) / 4 * 4;
  }
  PI_CUDA(ctx, cudaMemcpyAsync(m->meta.ptr, host, words * 4, cudaMemcpyHostToDevice, ctx->stream));
  const int32_t* d = static_cast<const int32_t*>(m->meta.ptr);
  pi_seq_batch& b = st->b;
  b.n_seqs = n;
  b.rows = rows;
  b.tokens = reinterpret_cast<const uint32_t*>(d + o_tok);
  b.row_seq = d + o_rs;
  b.row_pos = d + o_rp;
  b.seq_row0 = d + o_r0;
  b.seq_n = d + o_n;
  b.seq_start = d + o_st;
  b.slot = d + o_sl;
  b.lens = d + o_ln;
  b.tables = d + o_tb;
  b.max_blocks = in->max_blocks;
  b.single_rows = d + o_si;
  b.n_single = (int)single.size();
  b.portions = d + o_po;
  b.n_portions = (int)portions.size();
  b.max_portion = max_portion;
  b.scan_seqs = d + o_sc;
  b.n_scan = (int)scan.size();
  b.chunk_seqs = d + o_cs;
  b.n_chunk_seqs = (int)chunk_seqs.size();
  b.chunks = d + o_ch;
  b.n_chunks = (int)chunks.size() / 2;
  b.chunk0 = d + o_c0;
  b.max_pos = max_pos + extra_positions;
  st->out_rows = d + o_out;
  st->n_out = in->n_out;
  // scratch is sized here, so that nothing allocates while a step is being captured
  size_t floats = 0;
  for (const Layer& L : m->layers)
    if (L.attn < 0) floats = std::max(floats, pi_recurrence_scratch_floats(L.rec, b.n_chunks));
  if (floats) PI_TRY(pi_reserve(ctx, &m->scratch, floats * sizeof(float)));
  if (in->n_out) {
    PI_TRY(pi_reserve(ctx, &m->head_in, (size_t)in->n_out * m->ld_h * sizeof(float)));
    PI_TRY(pi_reserve(ctx, &m->logits, (size_t)in->n_out * m->c.vocab_size * sizeof(float)));
    PI_TRY(pi_reserve(ctx, &m->ids, (size_t)in->n_out * sizeof(uint32_t)));
  }
  if (m->trace_on) PI_TRY(pi_reserve(ctx, &m->trace, m->layers.size() * m->c.max_rows * m->c.width * sizeof(float)));
  return PI_OK;
}

pi_status project(pi_ctx* ctx, const pi_linear* lin, const void* in, size_t in_ld, int M, bool bf16, pi_linear_args a) {
  a.M = M;
  a.x_stride = in_ld;
  if (bf16) {
    a.x_bf16 = static_cast<const __nv_bfloat16*>(in);
    return pi_launch_gemm_bf16(ctx, lin, a);
  }
  a.x = static_cast<const float*>(in);
  return pi_launch_gemv(ctx, lin, a);
}

pi_status run_layers(pi_ctx* ctx, pi_layered* m, pi_kv_pool* pool, pi_state_pool* state, const Staged& st) {
  const pi_seq_batch& b = st.b;
  const int M = b.rows, W = m->c.width, NL = (int)m->layers.size();
  const bool bf16 = act_bf16(ctx, m, M);
  const int kind = bf16 ? PI_BF16 : PI_F32;
  {
    pi_prof_scope prof(ctx, PI_PROF_OTHER);
    auto k = bf16 ? embed_dyt_kernel<__nv_bfloat16> : embed_dyt_kernel<float>;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(M), dim3(256), 0, 1, static_cast<const uint16_t*>(m->embed->w), m->embed->ld,
                                    m->c.vocab_size, W, b.tokens, m->x, m->layers[0].norm1, m->h, m->ld_h));
  }
  for (int i = 0; i < NL; ++i) {
    const Layer& L = m->layers[i];
    const pi_layer_config& c = L.c;
    const pi_dyt after = i + 1 < NL ? m->layers[i + 1].norm1 : m->final_norm;
    pi_linear_args in;
    in.out = m->proj;
    in.out_stride = m->ld_proj;
    if (c.mixer == PI_MIXER_ATTENTION) {
      const pi_kv_region& g = pool->regions[L.attn];
      pi_kv_view kv;
      kv.base = reinterpret_cast<char*>(pool->data) + g.offset;
      kv.kind = pool->kind;
      kv.kv_heads = g.kv_heads;
      kv.maps = g.maps;
      kv.dp = g.dp;
      kv.vp = g.vp;
      kv.block_size = pool->L.block_size;
      pi_maps_attention a;
      a.heads = c.heads;
      a.kv_heads = c.kv_heads;
      a.maps = c.maps;
      a.dim = c.dim;
      a.vdim = c.vdim;
      a.window = c.window;
      a.scale = c.scale;
      a.eps = m->c.norm_eps;
      a.lambda = L.lambda;
      a.out_scale = 1.0f - c.diff;
      a.rot_dims = c.rot_dims;
      a.rope_cos = m->ropes[L.rope].cos;
      a.rope_sin = m->ropes[L.rope].sin;
      pi_maps_kv mk;
      if (c.dim % 2 == 0) {   // rotary positions and the KV write fold into the projection
        mk.q_rows = c.heads * c.maps * c.dim;
        mk.k_rows = c.kv_heads * c.maps * c.dim;
        mk.maps = c.maps;
        mk.dim = c.dim;
        mk.vdim = c.vdim;
        mk.rot_dims = c.rot_dims;
        mk.rope_cos = a.rope_cos;
        mk.rope_sin = a.rope_sin;
        mk.base = kv.base;
        mk.kind = kv.kind;
        mk.kv_heads = kv.kv_heads;
        mk.dp = kv.dp;
        mk.vp = kv.vp;
        mk.block_size = kv.block_size;
        mk.row_seq = b.row_seq;
        mk.row_pos = b.row_pos;
        mk.lens = b.lens;
        mk.tables = b.tables;
        mk.max_blocks = b.max_blocks;
        in.epi = PI_EPI_MAPS_QKV;
        in.maps_kv = &mk;
      }
      PI_TRY(project(ctx, L.in, m->h, m->ld_h, M, bf16, in));
      if (in.epi != PI_EPI_MAPS_QKV) PI_TRY(pi_launch_maps_rope_kv(ctx, a, kv, m->proj, m->ld_proj, b));
      PI_TRY(pi_launch_maps_attention(ctx, a, kv, m->proj, m->ld_proj, m->core, m->ld_core, kind, b));
    } else {
      PI_TRY(project(ctx, L.in, m->h, m->ld_h, M, bf16, in));
      pi_recurrence r = L.rec;
      r.state = state->data;
      r.state_stride = state->stride;
      PI_TRY(pi_launch_recurrence(ctx, r, m->proj, m->ld_proj, m->core, m->ld_core, kind, b, static_cast<float*>(m->scratch.ptr)));
    }
    pi_dyt_residual res;
    res.x = m->x;
    res.x_stride = W;
    res.post = L.norm1b;
    res.next = c.ff > 0 ? L.norm2 : after;
    res.h = m->h;
    res.h_stride = m->ld_h;
    {
      pi_linear_args a;
      a.epi = PI_EPI_DYT_RESIDUAL;
      a.residual = &res;
      PI_TRY(project(ctx, L.out, m->core, m->ld_core, M, bf16, a));
    }
    if (c.ff > 0) {
      pi_linear_args a;
      a.epi = PI_EPI_GEGLU;
      a.out = static_cast<float*>(m->ffh);
      a.out_bf16 = static_cast<__nv_bfloat16*>(m->ffh);
      a.out_stride = m->ld_ff;
      PI_TRY(project(ctx, L.gate_up, m->h, m->ld_h, M, bf16, a));
      res.post = L.norm2b;
      res.next = after;
      pi_linear_args d;
      d.epi = PI_EPI_DYT_RESIDUAL;
      d.residual = &res;
      PI_TRY(project(ctx, L.down, m->ffh, m->ld_ff, M, bf16, d));
    }
    if (m->trace_on)
      PI_CUDA(ctx, cudaMemcpyAsync(static_cast<float*>(m->trace.ptr) + (size_t)i * m->c.max_rows * W, m->x, (size_t)M * W * sizeof(float),
                                   cudaMemcpyDeviceToDevice, ctx->stream));
  }
  if (st.n_out == 0) return PI_OK;
  // the last epilogue left the final norm of every row in h; anything but all rows in order is gathered from x
  const bool head_bf16 = act_bf16(ctx, m, st.n_out);
  const void* last = m->h;
  if (!(st.all_rows && head_bf16 == bf16)) {
    pi_prof_scope prof(ctx, PI_PROF_OTHER);
    auto k = head_bf16 ? gather_dyt_kernel<__nv_bfloat16> : gather_dyt_kernel<float>;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(st.n_out), dim3(256), 0, 1, (const float*)m->x, W, st.out_rows, m->final_norm, m->head_in.ptr, m->ld_h));
    last = m->head_in.ptr;
  }
  pi_linear_args a;
  a.out = static_cast<float*>(m->logits.ptr);
  a.out_stride = m->c.vocab_size;
  return project(ctx, m->embed, last, m->ld_h, st.n_out, head_bf16, a);
}

pi_status multi_step(pi_ctx* ctx, pi_layered* m, pi_kv_pool* pool, pi_state_pool* state, const Staged& st, uint32_t* history, int* counter) {
  PI_TRY(run_layers(ctx, m, pool, state, st));
  uint32_t* ids = static_cast<uint32_t*>(m->ids.ptr);
  PI_TRY(pi_launch_argmax(ctx, static_cast<float*>(m->logits.ptr), m->c.vocab_size, st.n_out, m->c.vocab_size, ids));
  pi_prof_scope prof(ctx, PI_PROF_OTHER);
  PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, advance_seqs_kernel, dim3(1), dim3(256), 0, 1, const_cast<uint32_t*>(st.b.tokens), (const uint32_t*)ids, history,
                                  counter, const_cast<int32_t*>(st.b.row_pos), const_cast<int32_t*>(st.b.seq_start), st.b.n_seqs));
  return PI_OK;
}

}  // namespace

pi_status pi_layered_create(pi_ctx* ctx, const pi_layered_config* cfg, const pi_named_tensor* tensors, int n_tensors, int gla_rank,
                            uint64_t seed, float std, pi_layered** out) {
  *out = nullptr;
  PI_REQUIRE(ctx, ctx->tp == 1, "layered designs run on one GPU");
  PI_REQUIRE(ctx, cfg->width > 0 && cfg->vocab_size > 0 && cfg->num_layers > 0 && cfg->layers && cfg->max_rows > 0, "model config fields must be positive");
  PI_REQUIRE(ctx, cfg->compute == PI_BF16 || cfg->compute == PI_F32, "layered designs compute in bf16 or f32");
  PI_REQUIRE(ctx, tensors || gla_rank > 0, "synthetic weights need a rank for the decay's low-rank input");
  pi_layered* m = new (std::nothrow) pi_layered();
  if (!m) return pi_fail(ctx, PI_ERR_OOM, "host allocation failed");
  Loader ld;
  ld.ctx = ctx;
  ld.m = m;
  ld.synthetic = tensors == nullptr;
  ld.seed = seed;
  ld.std = std;
  for (int i = 0; i < n_tensors; ++i) ld.by_name[tensors[i].name] = &tensors[i];
  const pi_status s = build(ctx, cfg, ld, gla_rank, m);
  if (s != PI_OK) {
    pi_layered_destroy(m);
    return s;
  }
  *out = m;
  return PI_OK;
}

void pi_layered_destroy(pi_layered* m) {
  if (!m) return;
  if (m->step_exec) cudaGraphExecDestroy(m->step_exec);
  for (Layer& L : m->layers)
    for (pi_linear* l : {L.in, L.out, L.gate_up, L.down}) pi_linear_destroy(l);
  pi_linear_destroy(m->embed);
  for (RopeTable& t : m->ropes) {
    cudaFree(t.cos);
    cudaFree(t.sin);
  }
  for (void* p : m->owned) cudaFree(p);
  for (void* p : {(void*)m->x, (void*)m->proj, m->h, m->core, m->ffh, m->meta.ptr, m->head_in.ptr, m->logits.ptr, m->ids.ptr, m->scratch.ptr,
                  m->trace.ptr, m->history.ptr})
    if (p) cudaFree(p);
  delete m;
}

size_t pi_layered_weight_bytes(const pi_layered* m) { return m->weight_bytes; }
int pi_layered_max_rows(const pi_layered* m) { return m->c.max_rows; }
int pi_layered_vocab(const pi_layered* m) { return m->c.vocab_size; }
size_t pi_layered_state_floats(const pi_layered* m) { return m->state_floats; }

pi_status pi_layered_kv_regions(pi_ctx* ctx, const pi_layered* m, int num_blocks, int block_size, pi_kv_pool* pool) {
  const size_t es = m->c.compute == PI_BF16 ? 2 : 4;
  size_t at = 0;
  pool->kind = m->c.compute;
  for (const Layer& L : m->layers) {
    if (L.attn < 0) continue;
    pi_kv_region g;
    g.kv_heads = L.c.kv_heads;
    g.maps = L.c.maps;
    g.dp = (L.c.dim + 15) / 16 * 16;
    g.vp = (L.c.vdim + 15) / 16 * 16;
    g.block_bytes = (size_t)block_size * g.kv_heads * (g.maps * g.dp + g.vp) * es;
    g.offset = at;
    at += (g.block_bytes * num_blocks + 255) / 256 * 256;
    pool->regions.push_back(g);
  }
  pool->L = pi_kv_layout{(int)pool->regions.size(), num_blocks, block_size, 0, 0};
  pool->floats = at / sizeof(float);
  const cudaError_t e = cudaMalloc(&pool->data, std::max<size_t>(at, 256));
  if (e != cudaSuccess) return pi_fail(ctx, PI_ERR_OOM, "allocating a %.2f GiB KV pool: %s", at / 1073741824.0, cudaGetErrorString(e));
  PI_CUDA(ctx, cudaMemsetAsync(pool->data, 0, std::max<size_t>(at, 256), ctx->stream));
  return PI_OK;
}

pi_status pi_layered_step(pi_ctx* ctx, pi_layered* m, pi_kv_pool* pool, pi_state_pool* state, const pi_step_batch* batch, float* logits_host,
                          uint32_t* argmax_host) {
  Staged st;
  PI_TRY(stage(ctx, m, pool, state, batch, 0, &st));
  PI_TRY(run_layers(ctx, m, pool, state, st));
  if (st.n_out && argmax_host) {
    uint32_t* ids = static_cast<uint32_t*>(m->ids.ptr);
    PI_TRY(pi_launch_argmax(ctx, static_cast<float*>(m->logits.ptr), m->c.vocab_size, st.n_out, m->c.vocab_size, ids));
    PI_CUDA(ctx, cudaMemcpyAsync(argmax_host, ids, st.n_out * sizeof(uint32_t), cudaMemcpyDeviceToHost, ctx->stream));
  }
  if (st.n_out && logits_host)
    PI_CUDA(ctx, cudaMemcpyAsync(logits_host, m->logits.ptr, (size_t)st.n_out * m->c.vocab_size * sizeof(float), cudaMemcpyDeviceToHost, ctx->stream));
  return pi_ctx_synchronize(ctx);
}

pi_status pi_layered_step_multi(pi_ctx* ctx, pi_layered* m, pi_kv_pool* pool, pi_state_pool* state, const pi_step_batch* batch, int n_steps,
                                uint32_t* out_tokens_host) {
  PI_REQUIRE(ctx, n_steps > 0 && out_tokens_host && batch->n_seqs > 0 && batch->n_tokens, "bad arguments");
  for (int i = 0; i < batch->n_seqs; ++i) PI_REQUIRE(ctx, batch->n_tokens[i] == 1, "sequence %d brings more than one token", i);
  std::vector<int32_t> rows(batch->n_seqs);
  for (int i = 0; i < batch->n_seqs; ++i) rows[i] = i;
  pi_step_batch all = *batch;
  all.n_out = batch->n_seqs;
  all.out_rows = rows.data();
  Staged st;
  PI_TRY(stage(ctx, m, pool, state, &all, n_steps, &st));
  PI_TRY(pi_reserve(ctx, &m->history, 64 + (size_t)n_steps * batch->n_seqs * sizeof(uint32_t)));
  int* counter = static_cast<int*>(m->history.ptr);
  uint32_t* history = reinterpret_cast<uint32_t*>(static_cast<char*>(m->history.ptr) + 64);
  PI_CUDA(ctx, cudaMemsetAsync(counter, 0, 64, ctx->stream));
  // the first step runs eagerly (it sizes what is left to size), the others replay one captured step
  PI_TRY(multi_step(ctx, m, pool, state, st, history, counter));
  int done = 1;
  if (ctx->opt_graph && !ctx->prof_on && !m->trace_on && n_steps >= 4) {
    cudaGraph_t graph = nullptr;
    const uint64_t before = ctx->launches;
    cudaError_t e = cudaStreamBeginCapture(ctx->stream, cudaStreamCaptureModeThreadLocal);
    if (e == cudaSuccess) {
      const pi_status s = multi_step(ctx, m, pool, state, st, history, counter);
      e = cudaStreamEndCapture(ctx->stream, &graph);
      const uint64_t per_step = ctx->launches - before;
      ctx->launches = before;
      if (s == PI_OK && e == cudaSuccess && graph) {
        if (m->step_exec) {
          cudaGraphExecUpdateResultInfo info;
          if (cudaGraphExecUpdate(m->step_exec, graph, &info) != cudaSuccess) {
            cudaGetLastError();
            cudaGraphExecDestroy(m->step_exec);
            m->step_exec = nullptr;
          }
        }
        if (!m->step_exec) e = cudaGraphInstantiate(&m->step_exec, graph, 0);
        for (; e == cudaSuccess && done < n_steps; ++done) {
          e = cudaGraphLaunch(m->step_exec, ctx->stream);
          if (e == cudaSuccess) ctx->launches += per_step;
        }
      }
      if (graph) cudaGraphDestroy(graph);
      if (s != PI_OK) return s;
    }
    if (e != cudaSuccess) {
      cudaGetLastError();
      ctx->err = std::string("CUDA graph path unavailable: ") + cudaGetErrorString(e);
    }
  }
  for (; done < n_steps; ++done) PI_TRY(multi_step(ctx, m, pool, state, st, history, counter));
  PI_CUDA(ctx, cudaMemcpyAsync(out_tokens_host, history, (size_t)n_steps * batch->n_seqs * sizeof(uint32_t), cudaMemcpyDeviceToHost, ctx->stream));
  return pi_ctx_synchronize(ctx);
}

pi_status pi_layered_trace(pi_ctx* ctx, pi_layered* m, int on) {
  (void)ctx;
  m->trace_on = on != 0;
  return PI_OK;
}

pi_status pi_layered_read_layer(pi_ctx* ctx, const pi_layered* m, int layer, int rows, float* out) {
  PI_REQUIRE(ctx, m->trace_on && m->trace.ptr, "layers are not being traced");
  PI_REQUIRE(ctx, layer >= 0 && layer < (int)m->layers.size() && rows >= 1 && rows <= m->c.max_rows && out, "bad arguments");
  PI_CUDA(ctx, cudaMemcpyAsync(out, static_cast<const float*>(m->trace.ptr) + (size_t)layer * m->c.max_rows * m->c.width,
                               (size_t)rows * m->c.width * sizeof(float), cudaMemcpyDeviceToHost, ctx->stream));
  return pi_ctx_synchronize(ctx);
}

// ---- state pool ---------------------------------------------------------------------------------------------------------
extern "C" {

void pi_state_pool_destroy(pi_state_pool* pool) {
  if (!pool) return;
  if (pool->data) cudaFree(pool->data);
  delete pool;
}

size_t pi_state_pool_bytes(const pi_state_pool* pool) { return pool ? pool->stride * pool->slots * sizeof(float) : 0; }

pi_status pi_state_pool_create(pi_ctx* ctx, const pi_model* model, int num_slots, pi_state_pool** out) {
  PI_ENTER(ctx);
  PI_REQUIRE(ctx, model && out, "null pointer");
  *out = nullptr;
  const size_t floats = pi_model_state_bytes(model) / sizeof(float);
  PI_REQUIRE(ctx, floats > 0, "this model has no recurrent state");
  PI_REQUIRE(ctx, num_slots > 0, "a state pool needs at least one slot");
  pi_state_pool* p = new (std::nothrow) pi_state_pool();
  if (!p) return pi_fail(ctx, PI_ERR_OOM, "host allocation failed");
  p->stride = floats;
  p->slots = num_slots;
  const cudaError_t e = cudaMalloc(&p->data, floats * num_slots * sizeof(float));
  if (e != cudaSuccess) {
    delete p;
    return pi_fail(ctx, PI_ERR_OOM, "allocating %d state slots of %zu bytes: %s", num_slots, floats * sizeof(float), cudaGetErrorString(e));
  }
  *out = p;
  return PI_OK;
}

pi_status pi_state_copy_slot(pi_ctx* ctx, pi_state_pool* pool, int32_t src, int32_t dst) {
  PI_ENTER(ctx);
  PI_REQUIRE(ctx, pool && src != dst && src >= 0 && dst >= 0 && src < pool->slots && dst < pool->slots, "state slot %d -> %d", src, dst);
  PI_CUDA(ctx, cudaMemcpyAsync(pool->data + (size_t)dst * pool->stride, pool->data + (size_t)src * pool->stride, pool->stride * sizeof(float),
                               cudaMemcpyDeviceToDevice, ctx->stream));
  return PI_OK;
}

}  // extern "C"
