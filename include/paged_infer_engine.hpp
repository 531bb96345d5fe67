// The engine's step loop over the device library, restated in C++17 (header only): what Engine::step does in the
// reference (src/engine.rs:485-839) with greedy sampling and no speculation -
//
//   admit    waiting requests while the KV pool can house them: map the longest cached prefix, prefill only what
//            the cache did not cover (the last prompt token is always recomputed for its logits), publish the
//            prompt's blocks, fork extra samples (src/engine.rs:496-586)
//   advance  settle memory for every live sequence first (grow the mapping, split shared blocks copy-on-write:
//            src/engine.rs:612-699), then advance all of them with ONE batched call and commit the chosen tokens
//   reclaim  release finished sequences (their cached prompt blocks stay resident for later requests)
//
// With EngineConfig::mixed_batches a prompt is not prefilled at admission: its portions ride in the batched call of the
// step beside the tokens of the sequences that already decode.
//
// The KV pool lives on the device (pi_kv_pool), block bookkeeping is pi::mem::KvCacheManager, and every forward pass is
// pi_model_step, whatever the model: portions of prompts and single tokens, with the greedy choice made on the device
// (only token ids come back).  Models that carry recurrent state get a state pool, and each sequence a slot of it.
//
// feed() drives the same batched call with given tokens instead of sampled ones and hands back logits (replaying a
// recorded schedule); such sequences live beside the scheduled ones until end().
#pragma once
#include <cstdint>
#include <cstring>
#include <deque>
#include <map>
#include <string>
#include <vector>

#include "paged_infer_cuda.h"
#include "paged_infer_memory.hpp"

namespace pi {

struct EngineConfig {
  size_t block_size = 16;
  size_t num_blocks = 256;
  size_t max_batch_size = 64;        // rows of one batched forward (BatchScratch capacity, src/engine.rs:210); more live
                                     // sequences than this are advanced in several passes per step
  size_t prefill_chunk_size = 32;
  uint32_t eos_token = 0xFFFFFFFFu;
  bool prefix_cache = true;
  bool mixed_batches = false;        // portions of prompts beside decoded tokens
  size_t state_slots = 0;            // models with recurrent state: live sequences at most (0: max_batch_size)
};

enum class FinishReason { None, Eos, Length, OutOfMemory };

struct Request {
  uint64_t id = 0;
  std::vector<uint32_t> tokens;
  size_t max_tokens = 16;
  size_t num_samples = 1;
};

struct Completion {
  uint64_t request_id = 0;
  size_t sequence_id = 0;
  std::vector<uint32_t> generated;
  FinishReason reason = FinishReason::None;
  size_t cached_prompt_tokens = 0;
};

// The next tokens of a sequence that is fed rather than sampled, and the places among them whose logits are wanted.
struct Feed {
  uint64_t id = 0;
  std::vector<uint32_t> tokens;
  std::vector<int32_t> want;
};

struct EngineStats {
  uint64_t steps = 0, requests = 0, prompt_tokens = 0, prompt_tokens_prefilled = 0, generated_tokens = 0, decode_batches = 0;
};

class EngineError : public std::runtime_error {
 public:
  explicit EngineError(const std::string& m) : std::runtime_error(m) {}
};

class Engine {
 public:
  // `ctx` and `model` stay owned by the caller; the engine owns the KV pool and the state pool.
  Engine(pi_ctx* ctx, pi_model* model, const EngineConfig& cfg) : ctx_(ctx), model_(model), cfg_(cfg), kv_(cfg.num_blocks, cfg.block_size) {
    kv_.with_prefix_cache(cfg.prefix_cache);
    if (cfg_.max_batch_size == 0) throw EngineError("max_batch_size must be at least 1");
    // one batched forward never exceeds what the model's scratch was built for
    const int cap = pi_model_max_batch(model_);
    if (cap > 0 && (size_t)cap < cfg_.max_batch_size) cfg_.max_batch_size = (size_t)cap;
    if (cfg_.prefill_chunk_size == 0) cfg_.prefill_chunk_size = 1;
    if (cap > 0 && (size_t)cap < cfg_.prefill_chunk_size) cfg_.prefill_chunk_size = (size_t)cap;
    check(pi_kv_pool_create_for_model(ctx_, model_, (int)cfg.num_blocks, (int)cfg.block_size, &pool_), "pi_kv_pool_create_for_model");
    if (pi_model_state_bytes(model_) > 0) {
      const size_t slots = cfg.state_slots ? cfg.state_slots : cfg_.max_batch_size;
      kv_.with_state_slots(slots);
      const pi_status s = pi_state_pool_create(ctx_, model_, (int)slots, &state_);
      if (s != PI_OK) {
        const std::string why = pi_last_error(ctx_);
        pi_kv_pool_destroy(pool_);
        throw EngineError("pi_state_pool_create: " + why);
      }
    }
  }
  // The uniform layout of the model is implied; kept for hosts that state it.
  Engine(pi_ctx* ctx, pi_model* model, const pi_kv_layout&, const EngineConfig& cfg) : Engine(ctx, model, cfg) {}
  ~Engine() {
    if (pool_) pi_kv_pool_destroy(pool_);
    if (state_) pi_state_pool_destroy(state_);
  }
  Engine(const Engine&) = delete;
  Engine& operator=(const Engine&) = delete;

  void add_request(Request r) {
    if (r.tokens.empty()) throw EngineError("a request needs at least one prompt token");
    if (r.num_samples == 0) r.num_samples = 1;
    if (state_ && r.num_samples > kv_.total_state_slots())
      throw EngineError("a request of this many samples never fits the state slots");
    waiting_.push_back(std::move(r));
  }
  bool has_work() const { return !waiting_.empty() || !active_.empty(); }
  size_t active_sequences() const { return active_.size(); }
  const EngineStats& stats() const { return stats_; }
  const mem::KvCacheManager& memory() const { return kv_; }
  std::vector<Completion> take_finished() {
    std::vector<Completion> out;
    out.swap(finished_);
    return out;
  }

  void step() {
    ++tick_;
    admit();
    advance();
    reclaim();
    ++stats_.steps;
  }

  // One batch of given tokens; logits: [total wanted][vocab], in the order of the entries and of their `want`.
  void feed(const std::vector<Feed>& entries, float* logits) {
    ++tick_;
    std::vector<Portion> batch;
    size_t rows = 0;
    for (const Feed& f : entries) {
      if (f.tokens.empty()) continue;
      auto it = fed_.find(f.id);
      if (it == fed_.end()) {
        const size_t seq = next_seq_++;
        auto adm = kv_.admit(seq, f.tokens, tick_, false);
        if (!adm) throw EngineError("no blocks or no state slot left for a new sequence");
        Sequence s;
        s.id = seq;
        s.request_id = f.id;
        s.table = std::move(adm->block_table);
        it = fed_.emplace(f.id, std::move(s)).first;
      }
      for (const Portion& p : batch)
        if (p.seq == &it->second) throw EngineError("a sequence appears twice in one step");
      batch.push_back(Portion{&it->second, f.tokens.data(), f.tokens.size(), it->second.length, f.want});
      rows += f.tokens.size();
    }
    if (rows > cfg_.max_batch_size) throw EngineError("the step brings more tokens than one batch takes");
    for (Portion& p : batch) {
      if (!settle(*p.seq, p.start, p.n)) throw EngineError("no block left for a fed sequence");
      p.seq->length += p.n;
    }
    if (!batch.empty()) run(batch, logits, nullptr);
  }
  void end(uint64_t id) {
    auto it = fed_.find(id);
    if (it == fed_.end()) return;
    kv_.release_sequence(it->second.id);
    fed_.erase(it);
  }

 private:
  struct Sequence {
    size_t id = 0;
    uint64_t request_id = 0;
    std::vector<uint32_t> token_ids;   // prompt + generated
    std::vector<uint32_t> generated;
    size_t prompt_len = 0;
    size_t length = 0;                 // tokens that have been run (fed sequences, and prompts on their way)
    size_t max_tokens = 0, num_samples = 1;
    size_t cached_prompt_tokens = 0;
    mem::BlockTable table;
    FinishReason finished = FinishReason::None;
    bool prefilling() const { return length < prompt_len; }
  };
  struct Portion {
    Sequence* seq;
    const uint32_t* tokens;
    size_t n, start;
    std::vector<int32_t> want;   // places in the portion
  };

  void check(pi_status s, const char* what) {
    if (s != PI_OK) throw EngineError(std::string(what) + ": " + pi_last_error(ctx_));
  }

  // Map blocks for positions start .. start + n - 1 and make them privately writable; false when the pool has none left.
  bool settle(Sequence& s, size_t start, size_t n) {
    const size_t bs = cfg_.block_size, needed = (start + n + bs - 1) / bs;
    while (s.table.len() < needed)
      if (!kv_.append_block(s.id, s.table, tick_)) return false;
    for (size_t lb = start / bs; lb < needed; ++lb) {   // forked siblings map the same partial block: split before writing
      kv_.ensure_writable(s.id, s.table, lb * bs, [&](mem::PhysicalBlock src, mem::PhysicalBlock dst) {
        check(pi_kv_copy_block(ctx_, pool_, src, dst), "pi_kv_copy_block");
      });
      if (kv_.allocator().is_shared(s.table.slots()[lb].block)) return false;   // no block left to split into
    }
    kv_.touch(s.id, tick_);
    return true;
  }

  // The one batched forward: portions (memory settled) of any lengths, results of the wanted places in order.
  void run(const std::vector<Portion>& batch, float* logits, uint32_t* ids) {
    const size_t n = batch.size();
    size_t width = 1, base = 0;
    for (const Portion& p : batch) width = std::max(width, p.seq->table.len());
    std::vector<uint32_t> tokens;
    std::vector<int32_t> counts(n), starts(n), lens(n), slots(n, 0), tables(n * width, -1), rows;
    for (size_t i = 0; i < n; ++i) {
      const Portion& p = batch[i];
      tokens.insert(tokens.end(), p.tokens, p.tokens + p.n);
      counts[i] = (int32_t)p.n;
      starts[i] = (int32_t)p.start;
      lens[i] = (int32_t)p.seq->table.len();
      for (size_t j = 0; j < p.seq->table.len(); ++j) tables[i * width + j] = p.seq->table.slots()[j].block;
      if (state_) slots[i] = *kv_.state_slot(p.seq->id);
      for (int32_t w : p.want) {
        if (w < 0 || (size_t)w >= p.n) throw EngineError("a wanted place lies outside its portion");
        rows.push_back((int32_t)base + w);
      }
      base += p.n;
    }
    pi_step_batch b;
    memset(&b, 0, sizeof(b));
    b.n_seqs = (int32_t)n;
    b.tokens = tokens.data();
    b.n_tokens = counts.data();
    b.start_pos = starts.data();
    b.block_tables = tables.data();
    b.max_blocks = (int32_t)width;
    b.table_lens = lens.data();
    b.state_slots = state_ ? slots.data() : nullptr;
    b.n_out = (int32_t)rows.size();
    b.out_rows = rows.data();
    check(pi_model_step(ctx_, model_, pool_, state_, &b, logits, ids), "pi_model_step");
  }

  static void finish_if_done(Sequence& s, uint32_t chosen, uint32_t eos) {
    if (chosen == eos) s.finished = FinishReason::Eos;
    else if (s.generated.size() >= s.max_tokens || s.max_tokens <= 1) s.finished = FinishReason::Length;
  }
  void commit(Sequence& s, uint32_t chosen) {
    s.token_ids.push_back(chosen);
    s.generated.push_back(chosen);
    ++stats_.generated_tokens;
    finish_if_done(s, chosen, cfg_.eos_token);
  }

  void admit() {
    // Memory is the only gate, as in the reference (src/engine.rs:496-503): a request is admitted as soon as the pool
    // can house its prompt; the number of live sequences is not limited here (advance() takes them in passes).
    // All samples of one request are decoded greedily and therefore identical; the reference gives such requests a
    // temperature of 0.8 (src/engine.rs:543-551), and sampling beyond argmax stays with the host
    // (pi_model_decode_batch_rows hands back the logits of the sequences that need it).
    while (!waiting_.empty()) {
      const Request& req = waiting_.front();
      if (state_ && kv_.free_state_slots() < reserved_slots() + req.num_samples) break;   // samples need a slot each
      const size_t seq_id = next_seq_;
      auto adm = kv_.admit(seq_id, req.tokens, tick_);
      if (!adm) break;   // out of memory even after reclaiming cold cache blocks: wait for a live sequence to retire
      ++next_seq_;
      Sequence s;
      s.id = seq_id;
      s.request_id = req.id;
      s.token_ids = req.tokens;
      s.prompt_len = req.tokens.size();
      // replay only what the cache did not cover; a fully cached prompt still recomputes its last token for the logits
      s.length = std::min(adm->cached_tokens, req.tokens.size() - 1);
      s.max_tokens = req.max_tokens;
      s.num_samples = req.num_samples;
      s.cached_prompt_tokens = adm->cached_tokens;
      s.table = std::move(adm->block_table);
      ++stats_.requests;
      stats_.prompt_tokens += req.tokens.size();
      stats_.prompt_tokens_prefilled += req.tokens.size() - s.length;
      waiting_.pop_front();
      active_.push_back(std::move(s));
      if (!cfg_.mixed_batches) {
        const size_t at = active_.size() - 1;
        while (active_[at].prefilling()) {
          uint32_t first = 0;
          std::vector<Portion> one{next_portion(active_[at], cfg_.prefill_chunk_size)};
          run(one, nullptr, &first);
          ran_prompt(at, one[0].n, first);
        }
      }
    }
  }
  size_t reserved_slots() const {   // slots that samples of prompts still on their way will take
    size_t n = 0;
    for (const Sequence& s : active_)
      if (s.prefilling()) n += s.num_samples - 1;
    return n;
  }
  // The next tokens of a prompt (at most `limit`); only the end of the prompt has a result.
  static Portion next_portion(Sequence& s, size_t limit) {
    Portion p{&s, s.token_ids.data() + s.length, std::min(limit, s.prompt_len - s.length), s.length, {}};
    if (s.length + p.n == s.prompt_len) p.want.push_back((int32_t)p.n - 1);
    return p;
  }
  // A portion of sequence `at`'s prompt has run; at its end `first` is the first generated token.
  void ran_prompt(size_t at, size_t n, uint32_t first) {
    active_[at].length += n;
    if (active_[at].prefilling()) return;
    kv_.publish_prompt_blocks(active_[at].table);
    const size_t samples = active_[at].num_samples;
    for (size_t i = 1; i < samples; ++i) {   // extra samples map the parent's blocks; divergence is paid lazily
      Sequence c = active_[at];
      c.id = next_seq_++;
      c.table = kv_.fork(active_[at].table, c.id, tick_);
      if (state_) check(pi_state_copy_slot(ctx_, state_, *kv_.state_slot(active_[at].id), *kv_.state_slot(c.id)), "pi_state_copy_slot");
      commit(c, first);
      active_.push_back(std::move(c));
    }
    commit(active_[at], first);
  }

  void advance() {
    // settle memory first: the batched forward needs the block tables final
    std::vector<size_t> decode, prompts;
    for (size_t idx = 0; idx < active_.size(); ++idx) {
      Sequence& s = active_[idx];
      if (s.finished != FinishReason::None) continue;
      if (s.prefilling()) {
        prompts.push_back(idx);   // its blocks were mapped at admission
        continue;
      }
      if (!settle(s, s.token_ids.size() - 1, 1)) {
        s.finished = FinishReason::OutOfMemory;
        continue;
      }
      decode.push_back(idx);
    }
    // passes of at most max_batch_size rows, like run_groups (src/engine.rs:722-760); what is left of a pass after the
    // decoded tokens goes to portions of prompts, oldest first
    size_t next_decode = 0, next_prompt = 0;
    while (next_decode < decode.size() || next_prompt < prompts.size()) {
      std::vector<Portion> batch;
      std::vector<size_t> who;
      size_t rows = 0;
      for (; next_decode < decode.size() && rows < cfg_.max_batch_size; ++next_decode, ++rows) {
        Sequence& s = active_[decode[next_decode]];
        who.push_back(decode[next_decode]);
        batch.push_back(Portion{&s, &s.token_ids.back(), 1, s.token_ids.size() - 1, {0}});
      }
      const bool decoded = rows > 0;
      for (; next_prompt < prompts.size() && rows < cfg_.max_batch_size; ++next_prompt) {
        Sequence& s = active_[prompts[next_prompt]];
        who.push_back(prompts[next_prompt]);
        batch.push_back(next_portion(s, std::min(cfg_.prefill_chunk_size, cfg_.max_batch_size - rows)));
        rows += batch.back().n;
      }
      std::vector<uint32_t> chosen(batch.size());
      run(batch, nullptr, chosen.data());
      if (decoded) ++stats_.decode_batches;
      size_t got = 0;
      for (size_t i = 0; i < who.size(); ++i) {   // commit (a finished prompt may append to active_)
        const uint32_t id = batch[i].want.empty() ? 0 : chosen[got++];
        if (active_[who[i]].prefilling()) ran_prompt(who[i], batch[i].n, id);
        else commit(active_[who[i]], id);
      }
    }
  }

  void reclaim() {
    std::vector<Sequence> keep;
    for (auto& s : active_) {
      if (s.finished == FinishReason::None) {
        keep.push_back(std::move(s));
        continue;
      }
      kv_.release_sequence(s.id);
      Completion c;
      c.request_id = s.request_id;
      c.sequence_id = s.id;
      c.generated = std::move(s.generated);
      c.reason = s.finished;
      c.cached_prompt_tokens = s.cached_prompt_tokens;
      finished_.push_back(std::move(c));
    }
    active_.swap(keep);
  }

  pi_ctx* ctx_;
  pi_model* model_;
  EngineConfig cfg_;
  mem::KvCacheManager kv_;
  pi_kv_pool* pool_ = nullptr;
  pi_state_pool* state_ = nullptr;
  std::deque<Request> waiting_;
  std::vector<Sequence> active_;
  std::map<uint64_t, Sequence> fed_;
  std::vector<Completion> finished_;
  EngineStats stats_;
  uint64_t tick_ = 0;
  size_t next_seq_ = 0;
};

}  // namespace pi
