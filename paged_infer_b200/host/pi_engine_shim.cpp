// C ABI over the engine loop of include/paged_infer_engine.hpp (admission, mixed batches, block and state-slot
// bookkeeping, greedy generation, feeding of given tokens), so that a host in another language drives the same engine
// the C++ tests drive.  It calls the device library (libpaged_infer_cuda.so), whose context and model handles it is
// given.  Plain pointers and sizes only; an error returns -1 and leaves its text in pie_error().
#include <cstdint>
#include <cstring>
#include <string>

#include "../../include/paged_infer_engine.hpp"

struct pie_engine {
  pi::Engine engine;
  std::string error;
  std::deque<pi::Completion> finished;
  pie_engine(pi_ctx* c, pi_model* m, const pi::EngineConfig& cfg) : engine(c, m, cfg) {}
};

namespace {
thread_local std::string g_create_error;
template <typename F>
long guarded(pie_engine* e, F&& f) {
  try {
    return f();
  } catch (const std::exception& x) {
    e->error = x.what();
    return -1;
  }
}
}  // namespace

extern "C" {

pie_engine* pie_create(pi_ctx* ctx, pi_model* model, size_t block_size, size_t num_blocks, size_t max_batch, size_t prefill_chunk,
                       uint32_t eos, int prefix_cache, int mixed_batches, size_t state_slots) {
  try {
    pi::EngineConfig c;
    c.block_size = block_size;
    c.num_blocks = num_blocks;
    c.max_batch_size = max_batch;
    c.prefill_chunk_size = prefill_chunk;
    c.eos_token = eos;
    c.prefix_cache = prefix_cache != 0;
    c.mixed_batches = mixed_batches != 0;
    c.state_slots = state_slots;
    return new pie_engine(ctx, model, c);
  } catch (const std::exception& x) {
    g_create_error = x.what();
    return nullptr;
  }
}
void pie_destroy(pie_engine* e) { delete e; }
// e == NULL: why the last pie_create on this thread failed.
const char* pie_error(const pie_engine* e) { return e ? e->error.c_str() : g_create_error.c_str(); }

long pie_add_request(pie_engine* e, uint64_t id, const uint32_t* tokens, size_t n, size_t max_tokens, size_t samples) {
  return guarded(e, [&]() -> long {
    pi::Request r;
    r.id = id;
    r.tokens.assign(tokens, tokens + n);
    r.max_tokens = max_tokens;
    r.num_samples = samples;
    e->engine.add_request(std::move(r));
    return 0;
  });
}
// One engine step; 1 while there is work left, 0 when there is none.
long pie_step(pie_engine* e) {
  return guarded(e, [&]() -> long {
    e->engine.step();
    for (auto& c : e->engine.take_finished()) e->finished.push_back(std::move(c));
    return e->engine.has_work() ? 1 : 0;
  });
}
// The oldest finished sequence: its number of generated tokens, or -1 when there is none; with `tokens` (room for
// `cap`) it is taken off the queue.
long pie_next_finished(pie_engine* e, uint64_t* id, int* reason, uint32_t* tokens, size_t cap) {
  if (e->finished.empty()) return -1;
  const pi::Completion& c = e->finished.front();
  const long n = (long)c.generated.size();
  if (id) *id = c.request_id;
  if (reason) *reason = (int)c.reason;
  if (tokens) {
    std::memcpy(tokens, c.generated.data(), std::min(cap, (size_t)n) * sizeof(uint32_t));
    e->finished.pop_front();
  }
  return n;
}
// One batch of given tokens: n entries, their tokens and wanted places one after the other; logits [total wanted][vocab].
long pie_feed(pie_engine* e, int n, const uint64_t* ids, const int32_t* n_tokens, const uint32_t* tokens, const int32_t* n_want,
              const int32_t* want, float* logits) {
  return guarded(e, [&]() -> long {
    std::vector<pi::Feed> f((size_t)n);
    for (int i = 0; i < n; ++i) {
      f[i].id = ids[i];
      f[i].tokens.assign(tokens, tokens + n_tokens[i]);
      f[i].want.assign(want, want + n_want[i]);
      tokens += n_tokens[i];
      want += n_want[i];
    }
    e->engine.feed(f, logits);
    return 0;
  });
}
long pie_end(pie_engine* e, uint64_t id) {
  return guarded(e, [&]() -> long {
    e->engine.end(id);
    return 0;
  });
}
// out[0..6]: steps, requests, prompt tokens, of them prefilled, generated tokens, free blocks, free state slots.
void pie_stats(const pie_engine* e, uint64_t* out) {
  const pi::EngineStats& s = e->engine.stats();
  out[0] = s.steps;
  out[1] = s.requests;
  out[2] = s.prompt_tokens;
  out[3] = s.prompt_tokens_prefilled;
  out[4] = s.generated_tokens;
  out[5] = e->engine.memory().available_blocks();
  out[6] = e->engine.memory().free_state_slots();
}

}  // extern "C"
