// Layered designs: a decoder whose layers each name a token mixer - windowed attention with one or two softmax maps, latent
// attention, a gated linear recurrence (GLA), a matrix memory (mLSTM), a state-space recurrence (SSD), lightning attention, a
// gated recurrence of single channels (minGRU) - and, if they have one, a feed-forward: dense and gated, or routed experts.  Four
// ways of normalising:
//
//   Dynamic Tanh   x += dyt(norm1b, mixer(dyt(norm1, x)));    x += dyt(norm2b, ff(dyt(norm2, x)))
//   layer norm     x += ls1 mixer(ln(norm1, x));              x += ls2 ff(ln(norm2, x))
//   RMS norm       x += mu rms(norm1b, mixer(rms(norm1, x))); x += mu rms(norm2b, ff(rms(norm2, x)));
//                  x += mu rms(side, proj(gelu(gate x) * e)), e: the layer's part of the token's row of a table
//   norm of the sum  x = rms(norm1, keep x + g1 mixer(x));   x = rms(norm2, keep x + g2 ff(x)),  g = sigmoid(rg x + b) per channel
//
// A norm of the sum leaves nothing between x and the next sublayer's input; the rows of a sublayer gate ride behind those of the
// projection that reads the same input, and the row kernel applies it.
// With RMS norms the projection that ends a sublayer stores its result, and the row kernel behind it normalises that, adds it to
// the residual stream and writes the next sublayer's input, all with the row in registers.
// Layer norm needs the whole row: the projection that ends a sublayer adds its scaled result to the residual stream, and a
// row kernel writes the next sublayer's input (behind experts it also adds up their outputs).
// Dynamic Tanh needs no statistics, so all of it folds into the projection that ends a sublayer: its epilogue adds the
// normalised result to the f32 residual stream and hands on the normalised input of the next sublayer.  Per layer:
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
  pi_layer_norm ln1, ln2;                                  // also the RMS norms before the sublayers
  pi_layer_norm post1, post2, post_side;                   // ... and behind them, times residual_mult
  pi_linear *side_gate = nullptr, *side_proj = nullptr;
  const float *bias = nullptr, *slopes = nullptr, *sinks = nullptr;   // attention: see pi_maps_attention, pi_maps_prepare
  int col_gate = -1;                                       // column of the gate per head
  int temp = -1;                                           // index of its table of query factors
  const float *qk_norm = nullptr, *sigmoid_bias = nullptr;
  const float *gate1_b = nullptr, *gate2_b = nullptr;      // sublayer gates: biases and columns (of the mixer's projection, of `route`)
  int col_gate1 = 0, col_router = 0;
  float v_lambda = 0.f;
  bool v_first = false;
  const float *ls1 = nullptr, *ls2 = nullptr;
  // routed experts: gate_up holds [shared gate/up | router | shared gate of the token], down the shared expert's
  pi_linear *in = nullptr, *out = nullptr, *gate_up = nullptr, *down = nullptr;
  pi_linear *expert_in = nullptr, *expert_out = nullptr;   // stacks of all experts
  pi_linear *ukv = nullptr, *uk_t = nullptr;               // latent attention
  int attn = -1;                 // index of the KV region it reads, its own or another layer's
  int rope = -1;                 // index of its rotary table
  float lambda = 0.f;
  pi_recurrence rec;
  pi_latent_attention lat;
  pi_ssd ssd;
  pi_mingru gru;
  pi_moe moe;
};

struct RopeTable {
  int dims = 0, cap = 0;
  bool banded = false;
  double base = 1., factor = 1., original = 1., fast = 1., slow = 1.;
  float *cos = nullptr, *sin = nullptr;
};

struct TempTable {               // what queries are multiplied by, per position
  double coef = 0., every = 1.;
  int cap = 0;
  float* f = nullptr;
};

// Angle per position of every pair, and the factor of cos and sin.  With a factor above 1, pairs that turn less than `slow`
// times within `original` positions are slowed by it, pairs that turn more than `fast` times are left alone, with a linear
// ramp over the pair index in between.  Banded: the ramp runs over the number of turns, and cos and sin do not grow.
double rope_frequencies(const RopeTable& t, std::vector<double>* f) {
  f->resize(t.dims / 2);
  const bool stretched = t.factor != 1.0;
  if (stretched && t.banded) {
    for (int i = 0; i < t.dims / 2; ++i) {
      const double plain = pow(t.base, -2.0 * i / t.dims), turns = t.original * plain / (2.0 * M_PI);
      const double s = turns > t.fast ? 1.0 : turns < t.slow ? 0.0 : t.fast > t.slow ? (turns - t.slow) / (t.fast - t.slow) : 1.0;
      (*f)[i] = (1.0 - s) * plain / t.factor + s * plain;
    }
    return 1.0;
  }
  auto turns = [&](double n) { return t.dims * log(t.original / (2.0 * M_PI * n)) / (2.0 * log(t.base)); };
  const double lo = stretched ? std::max(floor(turns(t.fast)), 0.0) : 0.0, hi = stretched ? std::min(ceil(turns(t.slow)), t.dims - 1.0) : 0.0;
  for (int i = 0; i < t.dims / 2; ++i) {
    const double plain = pow(t.base, -2.0 * i / t.dims);
    const double ramp = stretched ? std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0) : 0.0;
    (*f)[i] = plain / t.factor * ramp + plain * (1.0 - ramp);
  }
  return stretched ? 0.1 * log(t.factor) + 1.0 : 1.0;
}

}  // namespace

struct pi_layered {
  pi_layered_config c;
  std::vector<Layer> layers;
  std::vector<RopeTable> ropes;
  std::vector<TempTable> temps;
  std::vector<void*> owned;      // device vectors
  pi_linear *embed = nullptr, *head = nullptr;   // head: null if tied
  pi_linear* side_embed = nullptr;
  pi_linear* pairs = nullptr;    // table of token pairs
  int regions = 0;               // of the KV pool
  size_t mix_stride = 0;         // values of a row that are mixed between layers
  pi_dyt final_norm;
  pi_layer_norm final_ln;        // its weight carries the logits' scale
  size_t weight_bytes = 0, state_floats = 0;
  bool chunked = false;          // every recurrent layer has a chunked kernel
  bool latent = false, expand = false;   // latent attention; its long portions are expanded
  int latent_window = 0;         // the widest (<= 0: everything before)
  // scratch for c.max_rows rows; activations are sized for f32 and hold bf16 on the tensor path
  float *x = nullptr, *proj = nullptr;
  void *h = nullptr, *core = nullptr, *ffh = nullptr;
  float *y = nullptr, *first_v = nullptr;   // RMS norm: a sublayer's result; values of the first layer that mixes them
  void* side_h = nullptr;
  size_t ld_side = 0;
  size_t ld_h = 0, ld_core = 0, ld_ff = 0, ld_proj = 0;
  // latent attention, state-space recurrence, experts
  void *lat_q = nullptr, *lat_o = nullptr;
  float* ssd_y = nullptr;
  float *route = nullptr, *shared = nullptr;
  void *moe_h = nullptr, *moe_act = nullptr, *moe_y = nullptr, *moe_ints = nullptr;
  size_t ld_route = 0, ld_act = 0;
  size_t max_pairs = 0;
  pi_buffer exp_keys, exp_pool;
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
    return upload(v, out);
  }
  pi_status upload(const std::vector<float>& v, const float** out) {
    float* d = nullptr;
    PI_CUDA(ctx, cudaMalloc(&d, std::max<size_t>(v.size(), 1) * sizeof(float)));
    m->owned.push_back(d);
    PI_CUDA(ctx, cudaMemcpy(d, v.data(), v.size() * sizeof(float), cudaMemcpyHostToDevice));
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
  pi_status layer_norm(const std::string& name, pi_layer_norm* out, float scale = 1.f) {
    std::vector<float> v;
    PI_TRY(vec(name, m->c.width, &v, 1.f));
    for (float& x : v) x *= scale;
    out->eps = m->c.norm_eps;
    return upload(v, &out->w);
  }
  // Times scale (one + stored weight).
  pi_status rms_norm(const std::string& name, pi_layer_norm* out, float one, float scale) {
    std::vector<float> v;
    PI_TRY(vec(name, m->c.width, &v, 1.f - one));
    for (float& x : v) x = scale * (one + x);
    out->eps = m->c.norm_eps;
    return upload(v, &out->w);
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
  // Every head's [dim][rank] block of a matrix turned round: [heads * rank][dim].
  pi_status transposed_heads(const std::string& name, size_t heads, size_t dim, size_t rank, pi_linear** out) {
    std::vector<Piece> p;
    std::vector<uint16_t> turned;
    pi_tensor t = {};
    if (synthetic) {
      PI_TRY(piece(name, heads * rank, dim, 0, 1, &p));
    } else {
      PI_TRY(piece(name, heads * dim, rank, 0, 1, &p));   // checks the shape
      const uint16_t* src = static_cast<const uint16_t*>(p[0].src.host->data);
      turned.resize(heads * dim * rank);
      for (size_t h = 0; h < heads; ++h)
        for (size_t d = 0; d < dim; ++d)
          for (size_t r = 0; r < rank; ++r) turned[(h * rank + r) * dim + d] = src[(h * dim + d) * rank + r];
      t = pi_tensor{PI_BF16, 0, (int64_t)(heads * rank), (int64_t)dim, turned.data(), nullptr};
      p[0].src.host = &t;
      p[0].src.rows = p[0].nrows = heads * rank;
      p[0].src.cols = dim;
    }
    PI_TRY(matrix(p, heads * rank, dim, out));
    PI_CUDA(ctx, cudaStreamSynchronize(ctx->stream));     // `turned` may go
    return PI_OK;
  }
  pi_status matrix(const std::vector<Piece>& pieces, size_t rows, size_t cols, pi_linear** out) {
    PI_TRY(build_linear(ctx, pieces, rows, cols, 0, out));
    m->weight_bytes += pi_linear_weight_bytes(*out);
    return PI_OK;
  }
};

pi_status check_layer(pi_ctx* ctx, int i, const pi_layer_config& c) {
  PI_REQUIRE(ctx, c.mixer >= PI_MIXER_ATTENTION && c.mixer <= PI_MIXER_MINGRU, "layer %d: unknown mixer %d", i, c.mixer);
  PI_REQUIRE(ctx, c.heads > 0 && c.dim > 0 && c.vdim > 0 && c.ff >= 0, "layer %d: sizes must be positive", i);
  if (c.mixer == PI_MIXER_ATTENTION) {
    PI_REQUIRE(ctx, c.kv_heads > 0 && c.heads % c.kv_heads == 0, "layer %d: %d heads do not share %d key/value heads", i, c.heads, c.kv_heads);
    PI_REQUIRE(ctx, c.maps == 1 || c.maps == 2, "layer %d: %d softmax maps", i, c.maps);
    PI_REQUIRE(ctx, c.rot_dims <= c.dim, "layer %d: %d rotary channels of %d", i, c.rot_dims, c.dim);
    PI_REQUIRE(ctx, c.maps == 1 || !(c.distance_bias || c.sink || c.head_gate), "layer %d: distance bias, sink and head gate belong to one softmax map", i);
    PI_REQUIRE(ctx, c.q_temp_every >= 0., "layer %d: queries grow every %g tokens", i, c.q_temp_every);
    PI_REQUIRE(ctx, !c.norm_qk || (c.maps == 1 && !c.biases && !c.unit_qk && !c.v_mix && c.q_temp_every == 0.),
               "layer %d: norms over whole projections go with nothing else between projection and rotation", i);
    PI_REQUIRE(ctx, !c.sigmoid_weights || (c.maps == 1 && !c.distance_bias && !c.sink), "layer %d: sigmoid weights go with one map and plain scores", i);
    PI_REQUIRE(ctx, c.kv_from == 0 || c.norm_qk, "layer %d: keys of another layer go with norms over whole projections", i);
  } else if (c.mixer == PI_MIXER_MINGRU) {
    PI_REQUIRE(ctx, c.heads == 1, "layer %d: this recurrence has one head", i);
  } else if (c.mixer == PI_MIXER_LATENT) {
    PI_REQUIRE(ctx, c.rank > 0, "layer %d: the latent needs channels", i);
  } else if (c.mixer == PI_MIXER_GLA) {
    PI_REQUIRE(ctx, c.tau != 0.f, "layer %d: tau is zero", i);
  } else if (c.mixer == PI_MIXER_MLSTM) {
    PI_REQUIRE(ctx, c.gate_cap > 0.f, "layer %d: gate_cap must be positive", i);
  } else if (c.mixer == PI_MIXER_LIGHTNING) {
    PI_REQUIRE(ctx, c.decay, "layer %d: no decays", i);
    for (int h = 0; h < c.heads; ++h) PI_REQUIRE(ctx, c.decay[h] >= 0. && c.decay[h] <= 1., "layer %d: a decay of %g", i, c.decay[h]);
  } else {
    PI_REQUIRE(ctx, c.groups > 0 && c.heads % c.groups == 0, "layer %d: %d heads do not form %d groups", i, c.heads, c.groups);
    PI_REQUIRE(ctx, c.norm_groups > 0 && (c.heads * c.vdim) % c.norm_groups == 0, "layer %d: %d channels do not form %d parts", i, c.heads * c.vdim, c.norm_groups);
    PI_REQUIRE(ctx, c.conv >= 1, "layer %d: the convolution needs taps", i);
  }
  if (c.mixer == PI_MIXER_ATTENTION || c.mixer == PI_MIXER_LATENT) {
    PI_REQUIRE(ctx, c.rot_dims >= 0 && c.rot_dims % 2 == 0, "layer %d: %d rotary channels", i, c.rot_dims);
    PI_REQUIRE(ctx, c.rot_dims == 0 || c.rot_base > 0.f, "layer %d: rotary base must be positive", i);
    PI_REQUIRE(ctx, c.rot_dims == 0 || c.rot_factor == 0.0 || c.rot_factor == 1.0 ||
                        (c.rot_factor > 0.0 && c.rot_original > 0.0 && c.rot_fast > 0.0 && c.rot_slow > 0.0 && c.rot_base != 1.f),
               "layer %d: rotary scaling constants must be positive", i);
  }
  if (c.ff > 0) {
    PI_REQUIRE(ctx, c.ff_kind >= PI_FF_GELU && c.ff_kind <= PI_FF_EXPERTS, "layer %d: unknown feed-forward %d", i, c.ff_kind);
    if (c.ff_kind == PI_FF_EXPERTS) {
      PI_REQUIRE(ctx, c.experts > 0 && c.expert_groups > 0 && c.experts % c.expert_groups == 0, "layer %d: %d experts do not form %d groups", i, c.experts,
                 c.expert_groups);
      PI_REQUIRE(ctx, c.keep_groups >= 1 && c.keep_groups <= c.expert_groups, "layer %d: %d groups of %d are kept", i, c.keep_groups, c.expert_groups);
      PI_REQUIRE(ctx, c.top >= 1 && c.top <= c.experts / c.expert_groups * c.keep_groups, "layer %d: %d experts per token", i, c.top);
      PI_REQUIRE(ctx, c.shared_ff >= 0, "layer %d: sizes must be positive", i);
      PI_REQUIRE(ctx, c.unit >= PI_UNIT_CLAMPED && c.unit <= PI_UNIT_RELU2 && c.score >= PI_SCORE_SIGMOID && c.score <= PI_SCORE_CHOSEN &&
                          (c.group_best == 1 || c.group_best == 2), "layer %d: unknown kind of experts", i);
      PI_REQUIRE(ctx, c.unit != PI_UNIT_RELU2 || c.shared_ff == 0, "layer %d: a shared expert has gated units", i);
    }
  }
  return PI_OK;
}

// Largest sizes of what a step needs beside the projections' outputs.
struct Extents {
  size_t in = 0, core = 1, ff = 1, lat_q = 0, lat_o = 0, inner = 0, route = 0, act = 0, top = 0, experts = 0;
  bool chunk = true;
  int attn = 0;
  std::vector<int> own;            // per layer: its KV region, -1: it has none of its own
};

int add_rope(pi_layered* m, const pi_layer_config& c) {
  RopeTable t;
  t.dims = c.rot_dims;
  t.base = c.rot_base;
  if (c.rot_factor != 0.0 && c.rot_factor != 1.0) {
    t.factor = c.rot_factor;
    t.original = c.rot_original;
    t.fast = c.rot_fast;
    t.slow = c.rot_slow;
    t.banded = c.rot_banded != 0;
  }
  for (size_t i = 0; i < m->ropes.size(); ++i) {
    const RopeTable& o = m->ropes[i];
    if (o.dims == t.dims && o.banded == t.banded && o.base == t.base && o.factor == t.factor && o.original == t.original && o.fast == t.fast && o.slow == t.slow) return (int)i;
  }
  m->ropes.push_back(t);
  return (int)m->ropes.size() - 1;
}

int add_temp(pi_layered* m, const pi_layer_config& c) {
  for (size_t i = 0; i < m->temps.size(); ++i)
    if (m->temps[i].coef == c.q_temp_coef && m->temps[i].every == c.q_temp_every) return (int)i;
  TempTable t;
  t.coef = c.q_temp_coef;
  t.every = c.q_temp_every;
  m->temps.push_back(t);
  return (int)m->temps.size() - 1;
}

// Attention with one map: what else a layer has beside q, k, v.
pi_status build_attention_options(pi_ctx* ctx, Loader& ld, int i, const std::string& mix, Layer& L) {
  pi_layered* m = ld.m;
  const pi_layer_config& c = L.c;
  const size_t nq = (size_t)c.heads * c.maps * c.dim, nk = (size_t)c.kv_heads * c.maps * c.dim, nv = (size_t)c.kv_heads * c.vdim;
  if (c.biases) {
    std::vector<float> all, part;
    const std::pair<const char*, size_t> parts[3] = {{"q.b", nq}, {"k.b", nk}, {"v.b", nv}};
    for (const auto& p : parts) {
      PI_TRY(ld.vec(mix + p.first, p.second, &part));
      all.insert(all.end(), part.begin(), part.end());
    }
    PI_TRY(ld.upload(all, &L.bias));
  }
  if (c.sink) PI_TRY(ld.dev_vec(mix + "sink", c.heads, &L.sinks));
  if (c.sigmoid_weights) PI_TRY(ld.dev_vec(mix + "pb", c.heads, &L.sigmoid_bias, -3.f));
  if (c.norm_qk) {
    std::vector<float> q, k;
    PI_TRY(ld.vec(mix + "q.norm", nq, &q, 1.f));
    if (c.kv_from == 0) PI_TRY(ld.vec(mix + "k.norm", nk, &k, 1.f));
    q.insert(q.end(), k.begin(), k.end());
    PI_TRY(ld.upload(q, &L.qk_norm));
  }
  if (c.distance_bias) {
    std::vector<float> s(c.heads);
    for (int h = 0; h < c.heads; ++h) s[h] = (float)exp2(-8.0 * (h + 1) / c.heads);
    PI_TRY(ld.upload(s, &L.slopes));
  }
  if (c.q_temp_every > 0.) L.temp = add_temp(m, c);
  if (c.v_mix) {
    L.v_first = m->mix_stride == 0;
    if (L.v_first) m->mix_stride = nv;
    PI_REQUIRE(ctx, m->mix_stride == nv, "layer %d: %zu value channels do not mix with the first layer's %zu", i, nv, m->mix_stride);
    if (!L.v_first) {
      std::vector<float> lambda;
      PI_TRY(ld.vec(mix + "vmix", 1, &lambda, 0.5f));
      L.v_lambda = lambda[0];
    }
  }
  return PI_OK;
}

pi_status build_mixer(pi_ctx* ctx, Loader& ld, int i, int gla_rank, Layer& L, Extents& x) {
  pi_layered* m = ld.m;
  const pi_layer_config& c = L.c;
  const size_t W = m->c.width, core = (size_t)c.heads * c.vdim;
  const std::string mix = "l" + std::to_string(i) + ".mix.";
  std::vector<Piece> p;
  size_t rows = 0;
  auto add = [&](const char* name, size_t n) -> pi_status {
    PI_TRY(ld.piece(mix + name, n, W, rows, 1, &p));
    rows += n;
    return PI_OK;
  };
  if (c.mixer == PI_MIXER_ATTENTION) {
    PI_TRY(add("q", (size_t)c.heads * c.maps * c.dim));
    if (c.kv_from > 0) {
      const int j = c.kv_from - 1;
      PI_REQUIRE(ctx, j < i && x.own[j] >= 0 && m->layers[j].c.mixer == PI_MIXER_ATTENTION, "layer %d: layer %d has no keys and values to share", i, j);
      const pi_layer_config& o = m->layers[j].c;
      PI_REQUIRE(ctx, o.kv_heads == c.kv_heads && o.maps == c.maps && o.dim == c.dim && o.vdim == c.vdim, "layer %d: its heads differ from those of layer %d", i, j);
      L.attn = x.own[j];
    } else {
      PI_TRY(add("k", (size_t)c.kv_heads * c.maps * c.dim));
      PI_TRY(add("v", (size_t)c.kv_heads * c.vdim));
      L.attn = x.own[i] = x.attn++;
    }
    PI_TRY(build_attention_options(ctx, ld, i, mix, L));
    if (c.head_gate) {
      L.col_gate = (int)rows;
      PI_TRY(add("g", c.heads));
    }
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
    L.rope = add_rope(m, c);
  } else if (c.mixer == PI_MIXER_LATENT) {
    pi_latent_attention& a = L.lat;
    a.heads = c.heads;
    a.dim = c.dim;
    a.rot_dims = c.rot_dims;
    a.vdim = c.vdim;
    a.rank = c.rank;
    a.window = c.window;
    a.scale = c.scale;
    a.eps = m->c.norm_eps;
    PI_TRY(add("q", (size_t)c.heads * (c.dim + c.rot_dims)));
    a.col_kv = (int)rows;
    PI_TRY(add("dkv", (size_t)c.rank + c.rot_dims));
    a.col_g = (int)rows;
    PI_TRY(add("g", core));
    PI_TRY(ld.dev_vec(mix + "dkv.norm", c.rank, &a.norm, 1.f));
    std::vector<Piece> u;
    PI_TRY(ld.piece(mix + "uk", (size_t)c.heads * c.dim, c.rank, 0, 1, &u));
    PI_TRY(ld.piece(mix + "uv", core, c.rank, (size_t)c.heads * c.dim, 1, &u));
    PI_TRY(ld.matrix(u, (size_t)c.heads * c.dim + core, c.rank, &L.ukv));
    PI_TRY(ld.transposed_heads(mix + "uk", c.heads, c.dim, c.rank, &L.uk_t));
    a.ukv = L.ukv;
    a.uk_t = L.uk_t;
    PI_REQUIRE(ctx, pi_latent_supported(ctx, a, m->c.compute), "layer %d: a latent of %d + %d channels is not supported", i, c.rank, c.rot_dims);
    L.attn = x.own[i] = x.attn++;
    L.rope = add_rope(m, c);
    if (!m->latent) {
      m->expand = true;
      m->latent_window = c.window;
    }
    m->latent = true;
    m->expand = m->expand && pi_latent_expandable(ctx, a, m->c.compute);
    m->latent_window = c.window <= 0 || m->latent_window <= 0 ? 0 : std::max(m->latent_window, c.window);
    x.lat_q = std::max(x.lat_q, (size_t)c.heads * pi_latent_dp(c.rank, c.rot_dims));
    x.lat_o = std::max(x.lat_o, (size_t)c.heads * c.rank);
  } else if (c.mixer == PI_MIXER_SSD) {
    pi_ssd& r = L.ssd;
    r.heads = c.heads;
    r.vdim = c.vdim;
    r.dim = c.dim;
    r.groups = c.groups;
    r.norm_groups = c.norm_groups;
    r.taps = c.conv;
    r.eps = m->c.norm_eps;
    r.col_x = (int)core;
    r.col_dt = (int)(core + r.channels());
    PI_TRY(add("in", core + r.channels() + c.heads));
    std::vector<float> taps;
    PI_TRY(ld.vec(mix + "conv", (size_t)r.channels() * c.conv, &taps, 0.25f));
    PI_TRY(ld.upload(taps, &r.conv));
    if (c.conv <= 4) {
      std::vector<float> four((size_t)r.channels() * 4, 0.f);
      for (int ch = 0; ch < r.channels(); ++ch)
        for (int j = 0; j < c.conv; ++j) four[(size_t)ch * 4 + 4 - c.conv + j] = taps[(size_t)ch * c.conv + j];
      const float* d;
      PI_TRY(ld.upload(four, &d));
      r.conv4 = reinterpret_cast<const float4*>(d);
    }
    PI_TRY(ld.dev_vec(mix + "conv.b", r.channels(), &r.conv_b));
    PI_TRY(ld.dev_vec(mix + "dt_bias", c.heads, &r.dt_bias, -2.f));
    PI_TRY(ld.dev_vec(mix + "A_log", c.heads, &r.a_log));
    PI_TRY(ld.dev_vec(mix + "D", c.heads, &r.d, 1.f));
    PI_TRY(ld.dev_vec(mix + "norm", core, &r.norm, 1.f));
    r.state_off = m->state_floats;
    m->state_floats += r.state_floats();
    x.inner = std::max(x.inner, core);
    x.chunk = x.chunk && pi_ssd_chunked(ctx, r, m->c.compute);
  } else if (c.mixer == PI_MIXER_LIGHTNING) {
    pi_ssd& r = L.ssd;               // keys are B, queries C, a group per head
    r.heads = r.groups = c.heads;
    r.vdim = c.vdim;
    r.dim = c.dim;
    r.eps = m->c.norm_eps;
    r.gate_last = true;
    r.col_x = (int)core;
    PI_TRY(add("g", core));
    PI_TRY(add("v", core));
    PI_TRY(add("k", (size_t)c.heads * c.dim));
    PI_TRY(add("q", (size_t)c.heads * c.dim));
    std::vector<float> decay(c.heads), log_decay(c.heads);
    for (int h = 0; h < c.heads; ++h) {
      decay[h] = (float)c.decay[h];
      log_decay[h] = (float)std::max(log(c.decay[h]), -1e4);   // a decay of 0 is one that leaves nothing
    }
    PI_TRY(ld.upload(decay, &r.decay));
    PI_TRY(ld.upload(log_decay, &r.log_decay));
    PI_TRY(ld.dev_vec(mix + "norm", core, &r.norm, 1.f));
    r.state_off = m->state_floats;
    m->state_floats += r.state_floats();
    x.inner = std::max(x.inner, core);
    x.chunk = x.chunk && pi_ssd_chunked(ctx, r, m->c.compute);
  } else if (c.mixer == PI_MIXER_MINGRU) {
    pi_mingru& r = L.gru;
    r.width = c.vdim;
    r.col_x = c.vdim;
    r.col_g = 2 * c.vdim;
    PI_TRY(add("z", core));
    PI_TRY(add("x", core));
    PI_TRY(add("g", core));
    PI_TRY(ld.dev_vec(mix + "z.b", core, &r.z_bias));
    PI_TRY(ld.dev_vec(mix + "x.b", core, &r.x_bias));
    r.state_off = m->state_floats;
    m->state_floats += r.state_floats();
  } else {
    pi_recurrence& r = L.rec;
    const size_t hd = (size_t)c.heads * c.dim;
    r.kind = c.mixer == PI_MIXER_GLA ? PI_REC_GLA : PI_REC_MLSTM;
    r.heads = c.heads;
    r.dim = c.dim;
    r.vdim = c.vdim;
    r.eps = m->c.norm_eps;
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
    x.chunk = x.chunk && pi_recurrence_chunked(ctx, r, m->c.compute);
  }
  if (m->c.sublayer_gate) {
    const std::string gate = "l" + std::to_string(i) + ".rg1";
    L.col_gate1 = (int)rows;
    PI_TRY(ld.piece(gate, W, W, rows, 1, &p));
    PI_TRY(ld.dev_vec(gate + ".b", W, &L.gate1_b));
    rows += W;
  }
  PI_TRY(ld.matrix(p, rows, W, &L.in));
  x.in = std::max(x.in, rows);
  x.core = std::max(x.core, core);
  p.clear();
  PI_TRY(ld.piece(mix + "o", W, core, 0, 1, &p));
  return ld.matrix(p, W, core, &L.out);
}

pi_status build_feed_forward(Loader& ld, int i, Layer& L, Extents& x) {
  const pi_layer_config& c = L.c;
  const size_t W = ld.m->c.width;
  const std::string mlp = "l" + std::to_string(i) + ".mlp.";
  std::vector<Piece> p;
  auto gated = [&](const std::string& name, size_t ff, size_t at) -> pi_status {   // interleaved gate and up rows
    PI_TRY(ld.piece(name + "gate", ff, W, at, 2, &p));
    return ld.piece(name + "up", ff, W, at + 1, 2, &p);
  };
  const size_t gate_rows = ld.m->c.sublayer_gate ? W : 0;
  auto sublayer_gate = [&](size_t at) -> pi_status {
    if (!gate_rows) return PI_OK;
    const std::string gate = "l" + std::to_string(i) + ".rg2";
    PI_TRY(ld.piece(gate, W, W, at, 1, &p));
    x.route = std::max(x.route, W);
    return ld.dev_vec(gate + ".b", W, &L.gate2_b);
  };
  if (c.ff_kind != PI_FF_EXPERTS) {
    PI_TRY(gated(mlp, c.ff, 0));
    PI_TRY(sublayer_gate(2 * (size_t)c.ff));
    PI_TRY(ld.matrix(p, 2 * (size_t)c.ff + gate_rows, W, &L.gate_up));
    p.clear();
    PI_TRY(ld.piece(mlp + "down", W, c.ff, 0, 1, &p));
    x.ff = std::max(x.ff, (size_t)c.ff);
    return ld.matrix(p, W, c.ff, &L.down);
  }
  pi_moe& e = L.moe;
  e.experts = c.experts;
  e.top = c.top;
  e.groups = c.expert_groups;
  e.keep = c.keep_groups;
  e.score = c.score;
  e.group_best = c.group_best;
  e.renorm = c.renorm;
  e.scale = c.route_scale;
  if (c.router_bias) PI_TRY(ld.dev_vec(mlp + "router.b", c.experts, &e.bias));
  else PI_TRY(ld.dev_vec(mlp + "correction", c.experts, &e.correction));
  size_t rows = 2 * (size_t)c.shared_ff;
  if (c.shared_ff) PI_TRY(gated(mlp + "shared.", c.shared_ff, 0));
  PI_TRY(sublayer_gate(rows));
  rows += gate_rows;
  L.col_router = (int)gate_rows;
  PI_TRY(ld.piece(mlp + "router", c.experts, W, rows, 1, &p));
  rows += c.experts;
  if (c.shared_ff && c.shared_gate) {
    PI_TRY(ld.piece(mlp + "shared.sg", 1, W, rows, 1, &p));
    ++rows;
  }
  PI_TRY(ld.matrix(p, rows, W, &L.gate_up));
  if (c.shared_ff) {
    p.clear();
    PI_TRY(ld.piece(mlp + "shared.down", W, c.shared_ff, 0, 1, &p));
    PI_TRY(ld.matrix(p, W, c.shared_ff, &L.down));
  }
  const size_t E = c.experts, ff = c.ff;
  p.clear();
  const bool unit_gated = c.unit != PI_UNIT_RELU2;
  for (size_t k = 0; k < E; ++k) {
    const std::string name = mlp + "e" + std::to_string(k) + ".";
    if (unit_gated) PI_TRY(gated(name, ff, k * 2 * ff));
    else PI_TRY(ld.piece(name + "up", ff, W, k * ff, 1, &p));
  }
  PI_TRY(ld.matrix(p, E * ff * (unit_gated ? 2 : 1), W, &L.expert_in));
  p.clear();
  for (size_t k = 0; k < E; ++k) PI_TRY(ld.piece(mlp + "e" + std::to_string(k) + ".down", W, ff, k * W, 1, &p));
  PI_TRY(ld.matrix(p, E * W, ff, &L.expert_out));
  x.ff = std::max(x.ff, (size_t)c.shared_ff);
  x.route = std::max(x.route, gate_rows + E + 1);
  x.act = std::max(x.act, ff);
  x.top = std::max(x.top, (size_t)c.top);
  x.experts = std::max(x.experts, E);
  return PI_OK;
}

pi_status build(pi_ctx* ctx, const pi_layered_config* cfg, Loader& ld, int gla_rank, pi_layered* m) {
  m->c = *cfg;
  m->c.layers = nullptr;
  const size_t W = cfg->width;
  const bool dyt = cfg->norm == PI_NORM_DYT, rms = cfg->norm == PI_NORM_RMS, of_sum = cfg->norm == PI_NORM_SUM;
  size_t tensors = 8;
  for (int i = 0; i < cfg->num_layers; ++i) tensors += 40 + 3 * (size_t)std::max(0, cfg->layers[i].experts);
  ld.keep.reserve(tensors);   // Source::host points into it
  Extents x;
  x.own.assign(cfg->num_layers, -1);
  {
    std::vector<Piece> p;
    PI_TRY(ld.piece("embed", cfg->vocab_size, W, 0, 1, &p));
    PI_TRY(ld.matrix(p, cfg->vocab_size, W, &m->embed));
    if (!cfg->tied) {
      p.clear();
      PI_TRY(ld.piece("head", cfg->vocab_size, W, 0, 1, &p));
      PI_TRY(ld.matrix(p, cfg->vocab_size, W, &m->head));
    }
  }
  if (cfg->side_dim > 0) {
    std::vector<Piece> p;
    const size_t cols = (size_t)cfg->side_dim * cfg->num_layers;
    PI_TRY(ld.piece("side.embed", cfg->vocab_size, cols, 0, 1, &p));
    PI_TRY(ld.matrix(p, cfg->vocab_size, cols, &m->side_embed));
  }
  if (cfg->pair_buckets > 0) {
    std::vector<Piece> p;
    PI_TRY(ld.piece("bigram", (size_t)cfg->pair_buckets + 1, W, 0, 1, &p));
    PI_TRY(ld.matrix(p, (size_t)cfg->pair_buckets + 1, W, &m->pairs));
    m->state_floats = 32;            // the previous token, in front of what the layers keep
  }
  if (dyt) PI_TRY(ld.dyt("final.norm", &m->final_norm));
  else if (of_sum) PI_TRY(ld.rms_norm("final.norm", &m->final_ln, 0.f, cfg->logit_scale));
  else if (rms) PI_TRY(ld.rms_norm("final.norm", &m->final_ln, 1.f, cfg->logit_scale));
  else PI_TRY(ld.layer_norm("final.norm", &m->final_ln, cfg->logit_scale));
  m->layers.resize(cfg->num_layers);
  for (int i = 0; i < cfg->num_layers; ++i) {
    Layer& L = m->layers[i];
    L.c = cfg->layers[i];
    PI_TRY(check_layer(ctx, i, L.c));
    PI_REQUIRE(ctx, !dyt || L.c.ff == 0 || L.c.ff_kind == PI_FF_GELU, "layer %d: this feed-forward is not built behind Dynamic Tanh", i);
    const std::string l = "l" + std::to_string(i);
    auto norm = [&](const char* name, pi_dyt* before, pi_dyt* after, pi_layer_norm* ln, pi_layer_norm* post, const char* scale_name,
                    const float** scale) -> pi_status {
      if (of_sum) return ld.rms_norm(l + name, post, 0.f, 1.f);
      if (rms) {
        PI_TRY(ld.rms_norm(l + name, ln, 1.f, 1.f));
        return ld.rms_norm(l + name + "b", post, 1.f, cfg->residual_mult);
      }
      if (dyt) {
        PI_TRY(ld.dyt(l + name, before));
        return ld.dyt(l + name + "b", after);
      }
      PI_TRY(ld.layer_norm(l + name, ln));
      return ld.dev_vec(l + scale_name, W, scale, 0.5f);
    };
    PI_TRY(norm(".norm1", &L.norm1, &L.norm1b, &L.ln1, &L.post1, ".ls1", &L.ls1));
    PI_TRY(build_mixer(ctx, ld, i, gla_rank, L, x));
    if (L.c.ff > 0) {
      PI_TRY(norm(".norm2", &L.norm2, &L.norm2b, &L.ln2, &L.post2, ".ls2", &L.ls2));
      PI_TRY(build_feed_forward(ld, i, L, x));
    }
    if (m->side_embed) {
      std::vector<Piece> p;
      PI_TRY(ld.piece(l + ".side.gate", cfg->side_dim, W, 0, 1, &p));
      PI_TRY(ld.matrix(p, cfg->side_dim, W, &L.side_gate));
      p.clear();
      PI_TRY(ld.piece(l + ".side.proj", W, cfg->side_dim, 0, 1, &p));
      PI_TRY(ld.matrix(p, W, cfg->side_dim, &L.side_proj));
      PI_TRY(ld.rms_norm(l + ".side.norm", &L.post_side, 0.f, cfg->residual_mult));
    }
    L.c.decay = nullptr;             // the caller's
  }
  m->chunked = x.chunk && m->state_floats > 0;
  m->regions = x.attn;
  const size_t cap = cfg->max_rows;
  m->ld_h = round8(W);
  m->ld_core = round8(x.core);
  m->ld_ff = round8(x.ff);
  m->ld_proj = round8(x.in);
  m->ld_route = round8(x.route);
  m->ld_act = round8(x.act);
  m->max_pairs = cap * x.top;
  auto alloc = [&](auto** p, size_t floats) -> pi_status {
    if (floats) PI_CUDA(ctx, cudaMalloc(p, floats * sizeof(float)));
    return PI_OK;
  };
  PI_TRY(alloc(&m->x, cap * W));
  PI_TRY(alloc(&m->proj, cap * m->ld_proj));
  PI_TRY(alloc(&m->h, cap * m->ld_h));
  PI_TRY(alloc(&m->core, cap * m->ld_core));
  PI_TRY(alloc(&m->ffh, cap * m->ld_ff));
  if (rms || of_sum) PI_TRY(alloc(&m->y, cap * W));
  PI_TRY(alloc(&m->first_v, cap * m->mix_stride));
  m->ld_side = round8(cfg->side_dim);
  PI_TRY(alloc(&m->side_h, cap * m->ld_side));
  const bool f32 = cfg->compute == PI_F32;
  PI_TRY(alloc(&m->lat_q, cap * x.lat_q / (f32 ? 1 : 2)));
  PI_TRY(alloc(&m->lat_o, (cap * x.lat_o + 1) / (f32 ? 1 : 2)));
  PI_TRY(alloc(&m->ssd_y, cap * x.inner));
  PI_TRY(alloc(&m->route, cap * m->ld_route));
  if (x.top) {
    PI_TRY(alloc(&m->shared, cap * W));
    PI_TRY(alloc(&m->moe_h, m->max_pairs * m->ld_h / 2));
    PI_TRY(alloc(&m->moe_act, m->max_pairs * m->ld_act));
    PI_TRY(alloc(&m->moe_y, m->max_pairs * W));
    // ids, weights, place, pair_at; then a tile (16 bytes) per pair at most
    PI_TRY(alloc(&m->moe_ints, 8 * m->max_pairs + 16));
  }
  PI_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  return PI_OK;
}

pi_moe_lists moe_lists(const pi_layered* m) {
  pi_moe_lists l;
  l.tiles = static_cast<int4*>(m->moe_ints);
  l.ids = reinterpret_cast<int32_t*>(l.tiles + m->max_pairs);
  l.weights = reinterpret_cast<float*>(l.ids + m->max_pairs);
  l.place = l.ids + 2 * m->max_pairs;
  l.pair_at = l.ids + 3 * m->max_pairs;
  l.n_tiles = l.ids + 4 * m->max_pairs;
  return l;
}

// Tables per position, grown to cover `positions`.
pi_status ensure_tables(pi_ctx* ctx, pi_layered* m, int positions) {
  for (TempTable& t : m->temps) {
    if (positions <= t.cap) continue;
    const int cap = std::max(positions, std::max(2 * t.cap, 2048));
    std::vector<float> f(cap);
    for (int p = 0; p < cap; ++p) f[p] = (float)(1.0 + t.coef * log(floor((p + 1) / t.every) + 1.0));
    PI_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    cudaFree(t.f);
    t.f = nullptr;
    t.cap = 0;
    PI_CUDA(ctx, cudaMalloc(&t.f, f.size() * sizeof(float)));
    PI_CUDA(ctx, cudaMemcpy(t.f, f.data(), f.size() * sizeof(float), cudaMemcpyHostToDevice));
    t.cap = cap;
  }
  for (RopeTable& t : m->ropes) {
    if (t.dims == 0 || positions <= t.cap) continue;
    const int cap = std::max(positions, std::max(2 * t.cap, 2048)), half = t.dims / 2;
    std::vector<float> c((size_t)cap * half), s(c.size());
    std::vector<double> f;
    const double gain = rope_frequencies(t, &f);
    for (int j = 0; j < half; ++j)
      for (int p = 0; p < cap; ++p) {
        c[(size_t)p * half + j] = (float)(gain * cos(p * f[j]));
        s[(size_t)p * half + j] = (float)(gain * sin(p * f[j]));
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
constexpr size_t kExpandBytes = (size_t)4 << 30;   // of the scratch pool for expanded keys and values

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
  PI_REQUIRE(ctx, pool && pool->regions.size() == (size_t)m->regions && pool->kind == m->c.compute,
             "the KV pool was made for another model");
  const int n = in->n_seqs;
  int rows = 0, max_pos = 0;
  std::vector<int32_t> row_seq, row_pos, row0(n), single, portions, scan, chunk_seqs, chunks, chunk0(1, 0);
  int max_portion = 0;
  std::vector<int32_t> latent_rows, expand, exp_lo, exp_start, exp_lens, exp_tables, key_seq, key_pos;
  int max_expand = 0, exp_max_blocks = 1, exp_blocks = 0;
  const int wide = m->latent_window;
  if (m->latent) {
    exp_lo.assign(n, 0);
    exp_start.assign(n, 0);
    exp_lens.assign(n, 0);
    size_t per_block = 0;
    for (const Layer& L : m->layers)
      if (L.c.mixer == PI_MIXER_LATENT) per_block = std::max(per_block, pi_latent_pool_elems(L.lat, 1) * sizeof(__nv_bfloat16));
    for (int i = 0; i < n && m->expand; ++i) {   // which portions are expanded, and what they see
      const int k = in->n_tokens[i], p0 = in->start_pos[i];
      if (k < kExpandPortion || k > m->c.max_rows || p0 < 0 || p0 >= (1 << 30)) continue;
      const int lo = wide > 0 ? std::max(0, p0 - wide + 1) / kExpandBlock * kExpandBlock : 0, blocks = (p0 + k - lo + kExpandBlock - 1) / kExpandBlock;
      if ((exp_blocks + blocks) * per_block > kExpandBytes) {   // all or none, so that a row's length tells its way
        expand.clear();
        exp_blocks = 0;
        break;
      }
      expand.push_back(i);
      exp_lo[i] = lo;
      exp_start[i] = p0 - lo;
      exp_lens[i] = blocks;
      exp_blocks += blocks;
      exp_max_blocks = std::max(exp_max_blocks, blocks);
      max_expand = std::max(max_expand, k);
    }
    exp_tables.assign((size_t)n * exp_max_blocks, 0);
    int next = 0;
    for (int i : expand) {
      for (int j = 0; j < exp_lens[i]; ++j) exp_tables[(size_t)i * exp_max_blocks + j] = next++;
      for (int t = 0; t < exp_start[i] + in->n_tokens[i]; ++t) {
        key_seq.push_back(i);
        key_pos.push_back(t);
      }
    }
  }
  for (int i = 0; i < n; ++i) {
    const int k = in->n_tokens[i], p0 = in->start_pos[i];
    PI_REQUIRE(ctx, k >= 1 && p0 >= 0 && p0 < (1 << 30), "sequence %d: %d tokens from position %d", i, k, p0);
    PI_REQUIRE(ctx, k <= m->c.max_rows - rows, "the step's tokens exceed the model's %d rows", m->c.max_rows);
    row0[i] = rows;
    for (int j = 0; j < k; ++j) {
      row_seq.push_back(i);
      row_pos.push_back(p0 + j);
    }
    if (m->latent && (expand.empty() || k < kExpandPortion))
      for (int j = 0; j < k; ++j) latent_rows.push_back(rows + j);
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
  PI_TRY(ensure_tables(ctx, m, max_pos + 1 + extra_positions));

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
               o_ch = put(chunks.data(), chunks.size()), o_c0 = put(chunk0.data(), chunk0.size()), o_out = put(in->out_rows, in->n_out),
               o_lr = put(latent_rows.data(), latent_rows.size()), o_ex = put(expand.data(), expand.size()), o_el = put(exp_lo.data(), exp_lo.size()),
               o_es = put(exp_start.data(), exp_start.size()), o_en = put(exp_lens.data(), exp_lens.size()),
               o_et = put(exp_tables.data(), exp_tables.size()), o_ks = put(key_seq.data(), key_seq.size()), o_kp = put(key_pos.data(), key_pos.size());
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
  b.latent_rows = d + o_lr;
  b.n_latent = (int)latent_rows.size();
  b.expand = d + o_ex;
  b.n_expand = (int)expand.size();
  b.max_expand = max_expand;
  b.exp_lo = d + o_el;
  b.exp_start = d + o_es;
  b.exp_lens = d + o_en;
  b.exp_tables = d + o_et;
  b.exp_max_blocks = exp_max_blocks;
  b.exp_blocks = exp_blocks;
  b.key_seq = d + o_ks;
  b.key_pos = d + o_kp;
  b.n_keys = (int)key_seq.size();
  st->out_rows = d + o_out;
  st->n_out = in->n_out;
  // scratch is sized here, so that nothing allocates while a step is being captured
  size_t floats = 0, keys = 0, elems = 0;
  for (const Layer& L : m->layers) {
    if (L.c.mixer == PI_MIXER_SSD || L.c.mixer == PI_MIXER_LIGHTNING) floats = std::max(floats, pi_ssd_scratch_floats(L.ssd, b.n_chunks));
    else if (L.c.mixer == PI_MIXER_GLA || L.c.mixer == PI_MIXER_MLSTM) floats = std::max(floats, pi_recurrence_scratch_floats(L.rec, b.n_chunks));
    else if (L.c.mixer == PI_MIXER_LATENT) {
      keys = std::max(keys, (size_t)b.n_keys * pi_latent_rp(L.c.rank));
      elems = std::max(elems, pi_latent_pool_elems(L.lat, b.exp_blocks));
    }
  }
  if (b.n_expand) {
    PI_TRY(pi_reserve(ctx, &m->exp_keys, keys * sizeof(__nv_bfloat16)));
    PI_TRY(pi_reserve(ctx, &m->exp_pool, elems * sizeof(__nv_bfloat16)));
  }
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

pi_kv_view kv_view(const pi_kv_pool* pool, int attn) {
  const pi_kv_region& g = pool->regions[attn];
  pi_kv_view kv;
  kv.base = reinterpret_cast<char*>(pool->data) + g.offset;
  kv.kind = pool->kind;
  kv.kv_heads = g.kv_heads;
  kv.maps = g.maps;
  kv.dp = g.dp;
  kv.vp = g.vp;
  kv.block_size = pool->L.block_size;
  return kv;
}

constexpr int kFoldRows = 128;

// The layer's mixer, from h to core.
pi_status run_mixer(pi_ctx* ctx, pi_layered* m, const Layer& L, pi_kv_pool* pool, pi_state_pool* state, const Staged& st, bool bf16) {
  const pi_seq_batch& b = st.b;
  const pi_layer_config& c = L.c;
  const int M = b.rows, kind = bf16 ? PI_BF16 : PI_F32;
  pi_linear_args in;
  in.out = m->proj;
  in.out_stride = m->ld_proj;
  if (c.mixer == PI_MIXER_ATTENTION) {
    const pi_kv_view kv = kv_view(pool, L.attn);
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
    a.slopes = L.slopes;
    a.sinks = L.sinks;
    a.sigmoid_bias = L.sigmoid_bias;
    if (c.head_gate) {
      a.gate = m->proj + L.col_gate;
      a.gate_stride = m->ld_proj;
      a.gate_per_head = true;
    }
    pi_maps_prepare prep;
    prep.norm_qk = L.qk_norm;
    prep.q_only = c.kv_from > 0;
    prep.bias = L.bias;
    prep.unit_qk = c.unit_qk != 0;
    prep.q_temp = L.temp >= 0 ? m->temps[L.temp].f : nullptr;
    if (c.v_mix) prep.mix = pi_value_mix{m->first_v, m->mix_stride, L.v_lambda, L.v_first};
    pi_maps_kv mk;
    // biases, rotary positions, temperature, value mixing and the KV write fold into the projection; what needs a whole head does not,
    // and where nothing is rotated a kernel of its own is faster for many rows than the look-ups in the epilogue
    if (c.dim % 2 == 0 && !c.unit_qk && !c.norm_qk && !c.head_gate && L.gate1_b == nullptr && (M <= kFoldRows || c.rot_dims > 0)) {
      mk.bias = prep.bias;
      mk.q_temp = prep.q_temp;
      mk.mix = prep.mix;
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
    if (in.epi != PI_EPI_MAPS_QKV) PI_TRY(pi_launch_maps_prepare(ctx, a, prep, kv, m->proj, m->ld_proj, b));
    return pi_launch_maps_attention(ctx, a, kv, m->proj, m->ld_proj, m->core, m->ld_core, kind, b);
  }
  PI_TRY(project(ctx, L.in, m->h, m->ld_h, M, bf16, in));
  if (c.mixer == PI_MIXER_LATENT) {
    pi_latent_attention a = L.lat;
    a.rope_cos = m->ropes[L.rope].cos;
    a.rope_sin = m->ropes[L.rope].sin;
    pi_latent_scratch s;
    s.q = m->lat_q;
    s.o = m->lat_o;
    s.keys = static_cast<__nv_bfloat16*>(m->exp_keys.ptr);
    s.pool = static_cast<__nv_bfloat16*>(m->exp_pool.ptr);
    return pi_launch_latent_attention(ctx, a, kv_view(pool, L.attn), m->proj, m->ld_proj, m->core, m->ld_core, kind, b, s);
  }
  if (c.mixer == PI_MIXER_MINGRU) {
    pi_mingru r = L.gru;
    r.state = state->data;
    r.state_stride = state->stride;
    return pi_launch_mingru(ctx, r, m->proj, m->ld_proj, m->core, m->ld_core, kind, b);
  }
  if (c.mixer == PI_MIXER_SSD || c.mixer == PI_MIXER_LIGHTNING) {
    pi_ssd r = L.ssd;
    r.state = state->data;
    r.state_stride = state->stride;
    return pi_launch_ssd(ctx, r, m->proj, m->ld_proj, m->ssd_y, m->core, m->ld_core, kind, b, static_cast<float*>(m->scratch.ptr));
  }
  pi_recurrence r = L.rec;
  r.state = state->data;
  r.state_stride = state->stride;
  return pi_launch_recurrence(ctx, r, m->proj, m->ld_proj, m->core, m->ld_core, kind, b, static_cast<float*>(m->scratch.ptr));
}

// The layer's experts, from h to *sum (which the row kernel that follows adds up).
pi_status run_experts(pi_ctx* ctx, pi_layered* m, const Layer& L, int M, bool bf16, pi_expert_sum* sum) {
  const pi_layer_config& c = L.c;
  const pi_moe_lists lists = moe_lists(m);
  const int pairs = M * c.top;
  const pi_epilogue unit = c.unit == PI_UNIT_SILU ? PI_EPI_SWIGLU : c.unit == PI_UNIT_RELU2 ? PI_EPI_RELU2 : PI_EPI_CLAMP_GLU;
  // the shared expert's first projection carries the rows of the sublayer gate and the router
  pi_linear_args a;
  if (c.shared_ff) {
    a.epi = unit;
    a.glu_limit = c.shared_limit;
    a.glu_rows = 2 * c.shared_ff;
    a.out = static_cast<float*>(m->ffh);
    a.out_bf16 = static_cast<__nv_bfloat16*>(m->ffh);
    a.out_stride = m->ld_ff;
    a.rest = m->route;
    a.rest_stride = m->ld_route;
  } else {
    a.out = m->route;
    a.out_stride = m->ld_route;
  }
  PI_TRY(project(ctx, L.gate_up, m->h, m->ld_h, M, bf16, a));
  PI_TRY(pi_launch_moe_route(ctx, L.moe, m->route + L.col_router, m->ld_route, M, lists));
  pi_expert_rows rows;
  rows.experts = c.experts;
  const void* x = m->h;
  if (bf16) {
    PI_TRY(pi_launch_moe_gather(ctx, L.moe, M, lists, static_cast<const __nv_bfloat16*>(m->h), m->ld_h, static_cast<__nv_bfloat16*>(m->moe_h)));
    rows.tiles = lists.tiles;
    rows.n_tiles = lists.n_tiles;
    rows.max_tiles = pi_moe_max_tiles(M, L.moe);
    rows.tile_rows = pi_moe_tile_rows(M, L.moe);
    x = m->moe_h;
  } else {
    rows.expert = lists.ids;
    rows.x_div = c.top;
  }
  pi_linear_args e;
  e.experts = &rows;
  e.epi = unit;
  e.glu_limit = c.limit;
  e.out = static_cast<float*>(m->moe_act);
  e.out_bf16 = static_cast<__nv_bfloat16*>(m->moe_act);
  e.out_stride = m->ld_act;
  PI_TRY(project(ctx, L.expert_in, x, m->ld_h, pairs, bf16, e));
  rows.x_div = 1;
  pi_linear_args d;
  d.experts = &rows;
  d.out = static_cast<float*>(m->moe_y);
  d.out_bf16 = bf16 ? static_cast<__nv_bfloat16*>(m->moe_y) : nullptr;
  d.out_stride = m->c.width;
  PI_TRY(project(ctx, L.expert_out, m->moe_act, m->ld_act, pairs, bf16, d));
  sum->top = c.top;
  sum->weights = lists.weights;
  sum->place = bf16 ? lists.place : nullptr;
  sum->y = m->moe_y;
  sum->y_bf16 = bf16;
  sum->y_stride = m->c.width;
  sum->scale = L.ls2;
  if (c.shared_ff) {
    pi_linear_args s;
    s.out = m->shared;
    s.out_stride = m->c.width;
    PI_TRY(project(ctx, L.down, m->ffh, m->ld_ff, M, bf16, s));
    sum->shared = m->shared;
    sum->shared_stride = m->c.width;
    if (c.shared_gate) {
      sum->shared_gate = m->route + L.col_router + c.experts;
      sum->shared_gate_stride = m->ld_route;
    }
  }
  return PI_OK;
}

// The layer's gated feed-forward, from h through the projection `down` describes.
pi_status run_dense(pi_ctx* ctx, pi_layered* m, const Layer& L, int M, bool bf16, const pi_linear_args& down) {
  pi_linear_args g;
  g.epi = L.c.ff_kind == PI_FF_SILU ? PI_EPI_SWIGLU : PI_EPI_GEGLU;
  g.out = static_cast<float*>(m->ffh);
  g.out_bf16 = static_cast<__nv_bfloat16*>(m->ffh);
  g.out_stride = m->ld_ff;
  if (L.gate2_b) {
    g.glu_rows = 2 * L.c.ff;
    g.rest = m->route;
    g.rest_stride = m->ld_route;
  }
  PI_TRY(project(ctx, L.gate_up, m->h, m->ld_h, M, bf16, g));
  return project(ctx, L.down, m->ffh, m->ld_ff, M, bf16, down);
}

// Layer i with RMS norms of the results or of the sums, from core, the mixer's heads, to `after`: the input of the next layer (or null for the last one's x alone).
pi_status run_sandwich(pi_ctx* ctx, pi_layered* m, const Layer& L, int i, const Staged& st, bool bf16, const pi_row_norm& row, const pi_row_norm& after) {
  const int M = st.b.rows;
  const pi_layer_config& c = L.c;
  const bool side = L.side_gate != nullptr;
  pi_linear_args a;                       // a sublayer's result
  a.out = m->y;
  a.out_stride = m->c.width;
  const bool of_sum = m->c.norm == PI_NORM_SUM;
  auto gate = [&](pi_row_norm* n, const float* z, size_t stride, const float* bias) {
    if (!bias) return;
    n->gate = z;
    n->gate_stride = stride;
    n->gate_bias = bias;
  };
  auto result = [&](const pi_row_norm& to, const pi_layer_norm& post) {
    pi_row_norm n = to;
    n.of_sum = of_sum;
    n.keep = m->c.residual_keep;
    n.y = m->y;
    n.y_stride = m->c.width;
    n.post = post;
    return n;
  };
  PI_TRY(project(ctx, L.out, m->core, m->ld_core, M, bf16, a));
  pi_row_norm n = result(side ? row : after, L.post1);   // the row step behind the last sublayer
  pi_expert_sum sum;
  if (c.ff > 0) {
    pi_row_norm between = result(row, L.post1);
    between.norm = L.ln2;            // null behind a norm of the sum: h is x as it stands
    gate(&between, m->proj + L.col_gate1, m->ld_proj, L.gate1_b);
    PI_TRY(pi_launch_row_norm(ctx, between));
    n.post = L.post2;
    gate(&n, m->route, m->ld_route, L.gate2_b);
    if (c.ff_kind == PI_FF_EXPERTS) {
      PI_TRY(run_experts(ctx, m, L, M, bf16, &sum));
      n.y = nullptr;
      n.experts = &sum;
    } else {
      PI_TRY(run_dense(ctx, m, L, M, bf16, a));
    }
  } else {
    gate(&n, m->proj + L.col_gate1, m->ld_proj, L.gate1_b);
  }
  if (!side) return pi_launch_row_norm(ctx, n);
  pi_token_side t;
  t.gate = L.side_gate;
  t.proj = L.side_proj;
  t.post = L.post_side;
  t.table = pi_token_table{static_cast<const uint16_t*>(m->side_embed->w) + (size_t)i * m->c.side_dim, m->side_embed->ld, m->c.vocab_size, st.b.tokens};
  if (pi_token_side_usable(ctx, t, M, m->c.width)) {
    n.norm = after.norm;
    n.h = after.h;
    n.h_kind = after.h_kind;
    return pi_launch_token_side(ctx, t, n);
  }
  PI_TRY(pi_launch_row_norm(ctx, n));     // h: x as it stands
  pi_linear_args g;
  g.epi = PI_EPI_GELU_TABLE;
  g.out = static_cast<float*>(m->side_h);
  g.out_bf16 = static_cast<__nv_bfloat16*>(m->side_h);
  g.out_stride = m->ld_side;
  g.table = t.table;
  PI_TRY(project(ctx, L.side_gate, m->h, m->ld_h, M, bf16, g));
  PI_TRY(project(ctx, L.side_proj, m->side_h, m->ld_side, M, bf16, a));
  return pi_launch_row_norm(ctx, result(after, L.post_side));
}

pi_status run_layers(pi_ctx* ctx, pi_layered* m, pi_kv_pool* pool, pi_state_pool* state, const Staged& st) {
  const pi_seq_batch& b = st.b;
  const int M = b.rows, W = m->c.width, NL = (int)m->layers.size();
  const bool bf16 = act_bf16(ctx, m, M), dyt = m->c.norm == PI_NORM_DYT, rms = m->c.norm == PI_NORM_RMS || m->c.norm == PI_NORM_SUM;
  const int kind = bf16 ? PI_BF16 : PI_F32;
  const bool head_bf16 = st.n_out && act_bf16(ctx, m, st.n_out);
  pi_row_norm row;               // layer or RMS norm: from x to h
  row.rms = rms;
  row.embed_scale = m->c.embed_scale;
  row.rows = M;
  row.width = W;
  row.x = m->x;
  row.h = m->h;
  row.ld_h = m->ld_h;
  row.h_kind = kind;
  if (dyt) {
    pi_prof_scope prof(ctx, PI_PROF_OTHER);
    auto k = bf16 ? embed_dyt_kernel<__nv_bfloat16> : embed_dyt_kernel<float>;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(M), dim3(256), 0, 1, static_cast<const uint16_t*>(m->embed->w), m->embed->ld,
                                    m->c.vocab_size, W, b.tokens, m->x, m->layers[0].norm1, m->h, m->ld_h));
  } else {
    pi_row_norm e = row;
    e.table = static_cast<const uint16_t*>(m->embed->w);
    e.table_ld = m->embed->ld;
    e.vocab = m->c.vocab_size;
    e.tokens = b.tokens;
    e.norm = m->layers[0].ln1;
    if (m->pairs)
      e.pairs = pi_token_pairs{static_cast<const uint16_t*>(m->pairs->w), m->pairs->ld, m->c.pair_buckets, m->c.pair_prev, m->c.pair_cur,
                               b.row_seq, b.seq_row0, b.seq_n, b.seq_start, b.slot, state->data, state->stride};
    PI_TRY(pi_launch_row_norm(ctx, e));
  }
  bool final_done = false;       // head_in holds the normalised rows
  for (int i = 0; i < NL; ++i) {
    const Layer& L = m->layers[i];
    const pi_layer_config& c = L.c;
    const bool last = i + 1 == NL;
    PI_TRY(run_mixer(ctx, m, L, pool, state, st, bf16));
    if (dyt) {
      const pi_dyt after = last ? m->final_norm : m->layers[i + 1].norm1;
      pi_dyt_residual res;
      res.x = m->x;
      res.x_stride = W;
      res.post = L.norm1b;
      res.next = c.ff > 0 ? L.norm2 : after;
      res.h = m->h;
      res.h_stride = m->ld_h;
      pi_linear_args a;
      a.epi = PI_EPI_DYT_RESIDUAL;
      a.residual = &res;
      PI_TRY(project(ctx, L.out, m->core, m->ld_core, M, bf16, a));
      if (c.ff > 0) {
        res.post = L.norm2b;
        res.next = after;
        PI_TRY(run_dense(ctx, m, L, M, bf16, a));
      }
    } else if (rms) {
      pi_row_norm after = row;
      if (!last) {
        after.norm = m->layers[i + 1].ln1;
      } else if (st.all_rows) {
        after.norm = m->final_ln;
        after.h = m->head_in.ptr;
        after.h_kind = head_bf16 ? PI_BF16 : PI_F32;
        final_done = true;
      } else {
        after.h = nullptr;
      }
      PI_TRY(run_sandwich(ctx, m, L, i, st, bf16, row, after));
    } else {
      pi_linear_args a;
      a.epi = PI_EPI_SCALE_ADD;
      a.out = m->x;
      a.out_stride = W;
      a.out_scale = L.ls1;
      PI_TRY(project(ctx, L.out, m->core, m->ld_core, M, bf16, a));
      pi_row_norm next = row;    // what the layer's end hands on; behind the last layer only the wanted rows are normalised
      if (!last) next.norm = m->layers[i + 1].ln1;
      else next.h = nullptr;
      if (c.ff > 0) {
        pi_row_norm n = row;
        n.norm = L.ln2;
        PI_TRY(pi_launch_row_norm(ctx, n));
      }
      pi_expert_sum sum;
      if (c.ff > 0 && c.ff_kind == PI_FF_EXPERTS) {
        PI_TRY(run_experts(ctx, m, L, M, bf16, &sum));
        next.experts = &sum;
        if (last && st.all_rows) {
          next.norm = m->final_ln;
          next.h = m->head_in.ptr;
          next.h_kind = head_bf16 ? PI_BF16 : PI_F32;
          final_done = true;
        }
      } else if (c.ff > 0) {
        a.out_scale = L.ls2;
        PI_TRY(run_dense(ctx, m, L, M, bf16, a));
      }
      if (next.h || next.experts) PI_TRY(pi_launch_row_norm(ctx, next));
    }
    if (m->trace_on)
      PI_CUDA(ctx, cudaMemcpyAsync(static_cast<float*>(m->trace.ptr) + (size_t)i * m->c.max_rows * W, m->x, (size_t)M * W * sizeof(float),
                                   cudaMemcpyDeviceToDevice, ctx->stream));
  }
  if (st.n_out == 0) return PI_OK;
  const void* last = m->head_in.ptr;
  if (!dyt) {
    if (!final_done) {
      pi_row_norm n = row;
      n.rows = st.n_out;
      n.pick = st.out_rows;
      n.norm = m->final_ln;
      n.h = m->head_in.ptr;
      n.h_kind = head_bf16 ? PI_BF16 : PI_F32;
      PI_TRY(pi_launch_row_norm(ctx, n));
    }
  } else if (!(st.all_rows && head_bf16 == bf16)) {
    // the last epilogue left the final norm of every row in h; anything but all rows in order is gathered from x
    pi_prof_scope prof(ctx, PI_PROF_OTHER);
    auto k = head_bf16 ? gather_dyt_kernel<__nv_bfloat16> : gather_dyt_kernel<float>;
    PI_LAUNCH_OK(ctx, pi_launch_dep(ctx, k, dim3(st.n_out), dim3(256), 0, 1, (const float*)m->x, W, st.out_rows, m->final_norm, m->head_in.ptr, m->ld_h));
  } else {
    last = m->h;
  }
  pi_linear_args a;
  a.out = static_cast<float*>(m->logits.ptr);
  a.out_stride = m->c.vocab_size;
  return project(ctx, m->head ? m->head : m->embed, last, m->ld_h, st.n_out, head_bf16, a);
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
  PI_REQUIRE(ctx, cfg->norm >= PI_NORM_DYT && cfg->norm <= PI_NORM_SUM, "unknown normalisation %d", cfg->norm);
  PI_REQUIRE(ctx, cfg->norm != PI_NORM_DYT || cfg->logit_scale == 1.f, "logits are not scaled behind Dynamic Tanh");
  PI_REQUIRE(ctx, cfg->side_dim >= 0, "sizes must be positive");
  PI_REQUIRE(ctx, cfg->norm == PI_NORM_RMS || (cfg->residual_mult == 1.f && cfg->side_dim == 0),
             "a factor of the residual update and a table of tokens belong to RMS norms of the results");
  PI_REQUIRE(ctx, cfg->norm == PI_NORM_SUM || (cfg->residual_keep == 1.f && !cfg->sublayer_gate), "sublayer gates and a factor of the residual stream belong to norms of the sum");
  PI_REQUIRE(ctx, cfg->norm >= PI_NORM_RMS || (cfg->embed_scale == 1.f && cfg->pair_buckets == 0), "a scale of the embedding and a table of token pairs belong to RMS norms");
  PI_REQUIRE(ctx, cfg->pair_buckets == 0 || (cfg->pair_buckets > 0 && cfg->pair_prev >= 0 && cfg->pair_prev < cfg->pair_buckets && cfg->pair_cur >= 0 &&
                                             cfg->pair_cur < cfg->pair_buckets), "the factors of a token pair are taken modulo the table's length");
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
    for (pi_linear* l : {L.in, L.out, L.gate_up, L.down, L.expert_in, L.expert_out, L.ukv, L.uk_t, L.side_gate, L.side_proj}) pi_linear_destroy(l);
  pi_linear_destroy(m->embed);
  pi_linear_destroy(m->head);
  pi_linear_destroy(m->side_embed);
  pi_linear_destroy(m->pairs);
  for (TempTable& t : m->temps) cudaFree(t.f);
  for (RopeTable& t : m->ropes) {
    cudaFree(t.cos);
    cudaFree(t.sin);
  }
  for (void* p : m->owned) cudaFree(p);
  for (void* p : {(void*)m->x, (void*)m->proj, m->h, m->core, m->ffh, m->lat_q, m->lat_o, (void*)m->ssd_y, (void*)m->route, (void*)m->shared, m->moe_h, m->moe_act,
                  m->moe_y, m->moe_ints, m->exp_keys.ptr, m->exp_pool.ptr, m->meta.ptr, m->head_in.ptr, m->logits.ptr, m->ids.ptr, m->scratch.ptr,
                  m->trace.ptr, (void*)m->y, (void*)m->first_v, m->side_h, m->history.ptr})
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
    if (L.attn < (int)pool->regions.size()) continue;   // none, or another layer's
    pi_kv_region g;
    if (L.c.mixer == PI_MIXER_LATENT) {   // [latent | rotated key part], common to the heads
      g.kv_heads = g.maps = 1;
      g.dp = pi_latent_dp(L.c.rank, L.c.rot_dims);
    } else {
      g.kv_heads = L.c.kv_heads;
      g.maps = L.c.maps;
      g.dp = (L.c.dim + 15) / 16 * 16;
      g.vp = (L.c.vdim + 15) / 16 * 16;
    }
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
