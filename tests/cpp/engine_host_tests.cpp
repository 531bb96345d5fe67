// The engine loop (include/paged_infer_engine.hpp) over a FAKE of the device library: the handful of C-ABI calls the
// engine makes are defined here on the host, so the scheduling logic runs without a GPU.  The fake "model" maps
// (last token, position) to the next token with a fixed formula, checks every argument the engine passes (batch
// rows within the model's capacity, block tables long enough for the position, distinct writable blocks after a
// copy-on-write) and records the batch sizes it saw.
//
// Scenarios (reference behaviour: Engine::admit src/engine.rs:496-586, run_groups :702-760):
//   oversize      a request with more samples than max_batch_size is admitted (memory is the only gate) and finishes
//   capacity      max_batch_size above the model's scratch capacity: every forward stays within the capacity
//   passes        more live sequences than max_batch_size: several passes per step, every sequence advances once
//   queue         a request that does not fit the pool waits without blocking the step loop from draining the others
#include <algorithm>
#include <cstdio>
#include <cstring>
#include <map>
#include <set>
#include <string>
#include <vector>

#include "../../include/paged_infer_engine.hpp"

struct pi_ctx { std::string err; };
struct pi_model { int capacity; size_t state_bytes = 0; };
struct pi_kv_pool { int num_blocks, block_size; };
struct FakeState { int next_pos = -1; uint32_t sum = 0; };   // what a recurrent model would carry
struct pi_state_pool { std::vector<FakeState> slots; };

static std::vector<int> g_batches;        // rows of every batched forward whose sequences bring one token each
static int g_mixed = 0;                   // forwards with portions of several tokens beside single ones
static int g_cow = 0, g_state_copies = 0;
static bool g_violation = false;

static uint32_t next_token(uint32_t tok, int pos) { return (tok * 31u + (uint32_t)pos * 7u + 3u) % 997u; }

extern "C" {
const char* pi_last_error(const pi_ctx* c) { return c ? c->err.c_str() : ""; }
int pi_model_max_batch(const pi_model* m) { return m->capacity; }
size_t pi_model_state_bytes(const pi_model* m) { return m->state_bytes; }
pi_status pi_kv_pool_create_for_model(pi_ctx*, const pi_model*, int num_blocks, int block_size, pi_kv_pool** out) {
  *out = new pi_kv_pool{num_blocks, block_size};
  return PI_OK;
}
void pi_kv_pool_destroy(pi_kv_pool* p) { delete p; }
pi_status pi_state_pool_create(pi_ctx*, const pi_model*, int n, pi_state_pool** out) {
  *out = new pi_state_pool{std::vector<FakeState>((size_t)n)};
  return PI_OK;
}
void pi_state_pool_destroy(pi_state_pool* p) { delete p; }
pi_status pi_state_copy_slot(pi_ctx*, pi_state_pool* p, int32_t src, int32_t dst) {
  if (src == dst) g_violation = true;
  p->slots.at(dst) = p->slots.at(src);
  ++g_state_copies;
  return PI_OK;
}
pi_status pi_kv_copy_block(pi_ctx* c, pi_kv_pool* p, int32_t src, int32_t dst) {
  if (src == dst || src < 0 || dst < 0 || src >= p->num_blocks || dst >= p->num_blocks) {
    c->err = "bad copy";
    return PI_ERR_INVALID_ARG;
  }
  ++g_cow;
  return PI_OK;
}
pi_status pi_model_step(pi_ctx* c, pi_model* m, pi_kv_pool* pool, pi_state_pool* state, const pi_step_batch* b, float* logits, uint32_t* argmax) {
  int rows = 0, singles = 0;
  for (int i = 0; i < b->n_seqs; ++i) {
    rows += b->n_tokens[i];
    singles += b->n_tokens[i] == 1;
  }
  if (rows > m->capacity) {
    c->err = "batch exceeds scratch capacity";
    return PI_ERR_INVALID_ARG;
  }
  if (singles == b->n_seqs) g_batches.push_back(b->n_seqs);
  else if (singles > 0) ++g_mixed;
  std::set<int32_t> written, slots;
  std::vector<uint32_t> out;
  const uint32_t* t = b->tokens;
  for (int i = 0; i < b->n_seqs; ++i) {
    const int first = b->start_pos[i] / pool->block_size, last = (b->start_pos[i] + b->n_tokens[i] - 1) / pool->block_size;
    if (last >= b->table_lens[i] || b->table_lens[i] > b->max_blocks) g_violation = true;
    else
      for (int lb = first; lb <= last; ++lb)
        if (!written.insert(b->block_tables[(size_t)i * b->max_blocks + lb]).second) g_violation = true;   // two sequences write one block
    if ((m->state_bytes > 0) != (b->state_slots != nullptr)) g_violation = true;
    FakeState* s = nullptr;
    if (m->state_bytes) {
      if (!slots.insert(b->state_slots[i]).second) g_violation = true;
      s = &state->slots.at(b->state_slots[i]);
      if (b->start_pos[i] == 0) *s = FakeState{0, 0};
      if (s->next_pos != b->start_pos[i]) g_violation = true;   // a slot was lost, shared or not carried on
    }
    for (int j = 0; j < b->n_tokens[i]; ++j, ++t) {
      uint32_t r = next_token(*t, b->start_pos[i] + j);
      if (s) {
        s->sum = s->sum * 13u + *t;
        s->next_pos = b->start_pos[i] + j + 1;
        r = (r + s->sum) % 997u;
      }
      out.push_back(r);
    }
  }
  for (int i = 0; i < b->n_out; ++i) {
    if (argmax) argmax[i] = out.at(b->out_rows[i]);
    if (logits) logits[i] = (float)out.at(b->out_rows[i]);
  }
  return PI_OK;
}
}

#define CHECK(cond)                                                  \
  do {                                                               \
    if (!(cond)) {                                                   \
      std::printf("FAILED %s:%d: %s\n", __FILE__, __LINE__, #cond);  \
      return 1;                                                      \
    }                                                                \
  } while (0)

static std::vector<uint32_t> prompt(uint32_t seed, size_t n) {
  std::vector<uint32_t> v;
  for (size_t i = 0; i < n; ++i) v.push_back((seed * 131u + (uint32_t)i * 17u) % 997u);
  return v;
}

static std::vector<uint32_t> expected(const std::vector<uint32_t>& p, size_t max_tokens) {
  std::vector<uint32_t> out;
  uint32_t tok = p.back();
  int pos = (int)p.size() - 1;
  while (out.size() < max_tokens) {
    tok = next_token(tok, pos++);
    out.push_back(tok);
  }
  return out;
}

static int run_all(pi::Engine& e, size_t want, std::map<uint64_t, std::vector<pi::Completion>>* done, int max_steps = 2000) {
  size_t got = 0;
  for (int s = 0; s < max_steps && e.has_work(); ++s) {
    e.step();
    for (auto& c : e.take_finished()) {
      (*done)[c.request_id].push_back(c);
      ++got;
    }
  }
  return (got == want && !e.has_work()) ? 0 : 1;
}

int main() {
  pi_ctx ctx;
  const pi_kv_layout L1 = {2, 1, 16, 2, 64};

  {  // oversize: 6 samples, max_batch_size 4 -> admitted, advanced in two passes per step, all complete
    g_batches.clear();
    pi_model model{64};
    pi::EngineConfig cfg;
    cfg.num_blocks = 64;
    cfg.max_batch_size = 4;
    pi::Engine e(&ctx, &model, L1, cfg);
    e.add_request({7, prompt(1, 20), 5, 6});
    e.add_request({8, prompt(2, 9), 3, 1});        // queued behind it: must not starve
    std::map<uint64_t, std::vector<pi::Completion>> done;
    CHECK(run_all(e, 7, &done) == 0);
    CHECK(done[7].size() == 6 && done[8].size() == 1);
    for (auto& c : done[7]) CHECK(c.generated == expected(prompt(1, 20), 5) && c.reason == pi::FinishReason::Length);
    CHECK(done[8][0].generated == expected(prompt(2, 9), 3));
    CHECK(*std::max_element(g_batches.begin(), g_batches.end()) <= 4);
    CHECK(g_cow >= 5);                             // the six siblings split their shared partial block
    std::printf("ok oversize\n");
  }
  {  // capacity: the engine is configured for 32 rows, the model's scratch holds 3
    g_batches.clear();
    pi_model model{3};
    pi::EngineConfig cfg;
    cfg.num_blocks = 64;
    cfg.max_batch_size = 32;
    pi::Engine e(&ctx, &model, L1, cfg);
    for (uint64_t r = 0; r < 8; ++r) e.add_request({r, prompt(10 + (uint32_t)r, 5 + r), 4, 1});
    std::map<uint64_t, std::vector<pi::Completion>> done;
    CHECK(run_all(e, 8, &done) == 0);
    for (uint64_t r = 0; r < 8; ++r) CHECK(done[r].size() == 1 && done[r][0].generated == expected(prompt(10 + (uint32_t)r, 5 + r), 4));
    CHECK(!g_batches.empty() && *std::max_element(g_batches.begin(), g_batches.end()) == 3);
    std::printf("ok capacity\n");
  }
  {  // passes: 10 live sequences, 4 rows per forward -> 3 forwards per step (4 + 4 + 2), every sequence advances once per step
    g_batches.clear();
    pi_model model{64};
    pi::EngineConfig cfg;
    cfg.num_blocks = 128;
    cfg.max_batch_size = 4;
    pi::Engine e(&ctx, &model, L1, cfg);
    for (uint64_t r = 0; r < 10; ++r) e.add_request({r, prompt(30 + (uint32_t)r, 18), 6, 1});
    e.step();
    CHECK(e.active_sequences() == 10);
    CHECK(g_batches.size() == 3 && g_batches[0] == 4 && g_batches[1] == 4 && g_batches[2] == 2);
    CHECK(e.stats().generated_tokens == 20);       // one token from each prefill, one from the step's decode
    std::map<uint64_t, std::vector<pi::Completion>> done;
    CHECK(run_all(e, 10, &done) == 0);
    for (uint64_t r = 0; r < 10; ++r) CHECK(done[r][0].generated == expected(prompt(30 + (uint32_t)r, 18), 6));
    std::printf("ok passes\n");
  }
  {  // queue: a prompt that needs more blocks than are free waits; the loop keeps draining the admitted ones
    pi_model model{64};
    pi::EngineConfig cfg;
    cfg.num_blocks = 6;
    cfg.max_batch_size = 8;
    cfg.prefix_cache = false;
    pi::Engine e(&ctx, &model, L1, cfg);
    e.add_request({1, prompt(50, 60), 3, 1});       // 4 blocks
    e.add_request({2, prompt(51, 60), 3, 1});       // 4 more: does not fit until request 1 retires
    e.step();
    CHECK(e.active_sequences() == 1);
    std::map<uint64_t, std::vector<pi::Completion>> done;
    CHECK(run_all(e, 2, &done) == 0);
    CHECK(done[1][0].generated == expected(prompt(50, 60), 3) && done[2][0].generated == expected(prompt(51, 60), 3));
    std::printf("ok queue\n");
  }
  // the same with recurrent state: tokens depend on everything before them
  auto expected_state = [](const std::vector<uint32_t>& p, size_t max_tokens) {
    std::vector<uint32_t> out, all = p;
    uint32_t sum = 0;
    size_t done = 0;
    while (out.size() < max_tokens) {
      for (; done < all.size(); ++done) sum = sum * 13u + all[done];
      out.push_back((next_token(all.back(), (int)all.size() - 1) + sum) % 997u);
      all.push_back(out.back());
    }
    return out;
  };
  for (int mixed = 0; mixed < 2; ++mixed) {   // slots: fewer than requests, given back and used again; samples copy the state
    g_mixed = g_state_copies = 0;
    pi_model model{24, 128};
    pi::EngineConfig cfg;
    cfg.num_blocks = 64;
    cfg.max_batch_size = 24;
    cfg.prefill_chunk_size = 7;
    cfg.mixed_batches = mixed != 0;
    cfg.state_slots = 4;
    pi::Engine e(&ctx, &model, cfg);
    for (uint64_t r = 0; r < 9; ++r) e.add_request({r, prompt(70 + (uint32_t)r % 4, 3 + 11 * r), 5 + r % 3, r == 4 ? 3u : 1u});
    std::map<uint64_t, std::vector<pi::Completion>> done;
    CHECK(run_all(e, 11, &done) == 0);
    for (uint64_t r = 0; r < 9; ++r)
      for (auto& c : done[r]) CHECK(c.generated == expected_state(prompt(70 + (uint32_t)r % 4, 3 + 11 * r), 5 + r % 3) && c.cached_prompt_tokens == 0);
    CHECK(g_state_copies == 2 && done[4].size() == 3 && (g_mixed > 0) == (mixed != 0));
    CHECK(e.memory().free_state_slots() == 4 && e.memory().available_blocks() == 64);
    std::printf("ok state slots (%s)\n", mixed ? "mixed batches" : "prefill at admission");
  }
  {  // mixed batches of a model without state: same tokens, the prefix cache still works
    pi_model model{16};
    pi::EngineConfig cfg;
    cfg.num_blocks = 64;
    cfg.max_batch_size = 16;
    cfg.prefill_chunk_size = 5;
    cfg.mixed_batches = true;
    pi::Engine e(&ctx, &model, cfg);
    for (uint64_t r = 0; r < 6; ++r) e.add_request({r, prompt(90, 40 + r), 6, 1});
    std::map<uint64_t, std::vector<pi::Completion>> done;
    CHECK(run_all(e, 6, &done) == 0);
    e.add_request({99, prompt(90, 40), 4, 1});
    CHECK(run_all(e, 1, &done) == 0);
    for (uint64_t r = 0; r < 6; ++r) CHECK(done[r][0].generated == expected(prompt(90, 40 + r), 6));
    CHECK(done[99][0].generated == expected(prompt(90, 40), 4) && done[99][0].cached_prompt_tokens == 32);
    std::printf("ok mixed batches\n");
  }
  {  // feed: given tokens in portions, results of the wanted places, slots and blocks used again after end()
    pi_model model{64, 64};
    pi::EngineConfig cfg;
    cfg.num_blocks = 6;
    cfg.state_slots = 2;
    cfg.prefix_cache = false;
    pi::Engine e(&ctx, &model, cfg);
    for (int round = 0; round < 3; ++round) {
      const auto a = prompt(5 + round, 40), b = prompt(15 + round, 30);
      auto sub = [](const std::vector<uint32_t>& v, size_t from, size_t to) { return std::vector<uint32_t>(v.begin() + from, v.begin() + to); };
      float out[4];
      e.feed({{1, sub(a, 0, 17), {}}}, out);
      e.feed({{1, sub(a, 17, 18), {}}, {2, sub(b, 0, 29), {3, 28}}}, out);
      CHECK(out[0] == (float)expected_state(sub(b, 0, 4), 1)[0] && out[1] == (float)expected_state(sub(b, 0, 29), 1)[0]);
      e.feed({{2, sub(b, 29, 30), {0}}, {1, sub(a, 18, 40), {21}}}, out);
      CHECK(out[0] == (float)expected_state(b, 1)[0] && out[1] == (float)expected_state(a, 1)[0]);
      bool full = false;
      try {
        e.feed({{3, prompt(1, 2), {0}}}, out);
      } catch (const pi::EngineError&) {
        full = true;
      }
      CHECK(full);
      e.end(1);
      e.end(2);
    }
    std::printf("ok feed\n");
  }
  bool threw = false;
  try {
    pi_model model{8};
    pi::EngineConfig cfg;
    cfg.max_batch_size = 0;
    pi::Engine e(&ctx, &model, L1, cfg);
  } catch (const pi::EngineError&) {
    threw = true;
  }
  CHECK(threw);
  CHECK(!g_violation);
  std::printf("all ok\n");
  return 0;
}
