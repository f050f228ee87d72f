// The engine over any model class: cache pages and state slots of live requests, ragged steps over
// them, and greedy generation with continuous batching. Host code only; it drives the model's own
// step. A slot is not cleared when it changes hands: a sequence's first token reads no state.
#include <algorithm>
#include <cstring>
#include <deque>
#include <unordered_map>

#include "model.h"

using namespace kanso;

namespace {
constexpr uint32_t MAX_STEP_TOKENS = 4096;  // rows of one model step (bounds the workspace)
constexpr uint32_t DEFAULT_STEP_TOKENS = 2048;
constexpr uint32_t NO_SLOT = 0xFFFFFFFFu;

struct Sequence {
  uint32_t len = 0;         // tokens in the cache
  uint32_t first_live = 0;  // table entries before it have gone back to the pool
  uint32_t slot = NO_SLOT;  // where its recurrent state lies, from its first step on
  std::vector<uint32_t> table;
};
// The next tokens of one sequence in a step.
struct Portion {
  Sequence* seq = nullptr;
  const uint32_t* tokens = nullptr;
  uint32_t n = 0;
};
}  // namespace

struct kanso_cuda_engine {
  kanso_cuda_model* model = nullptr;
  kanso_cuda_ctx* ctx = nullptr;
  kanso_cuda_kv* kv = nullptr;
  uint32_t block_size = 16, num_blocks = 0, max_seqs = 0;
  std::vector<uint32_t> free_blocks, free_slots;
  std::unordered_map<uint64_t, Sequence> live;
  uint32_t* d_next = nullptr;  // greedy tokens of a step
  size_t d_next_cap = 0;
  std::vector<uint32_t> tokens, query_lens, context_lens, tables, slots;  // host image of a step

  ~kanso_cuda_engine() {
    kanso_cuda_kv_destroy(kv);
    if (d_next) cudaFree(d_next);
  }

  // Pages for `n` more tokens of s and a state slot; nothing changes when there are too few.
  int32_t reserve(Sequence* s, uint32_t n) {
    const size_t need = ((uint64_t)s->len + n + block_size - 1) / block_size;
    const size_t more = need > s->table.size() ? need - s->table.size() : 0;
    if (more > free_blocks.size())
      return fail(ctx, KANSO_ERR_SHAPE, "engine: %zu more cache pages needed, %zu free", more,
                  free_blocks.size());
    if (s->slot == NO_SLOT) {
      if (free_slots.empty())
        return fail(ctx, KANSO_ERR_SHAPE, "engine: more than %u live requests", max_seqs);
      s->slot = free_slots.back();
      free_slots.pop_back();
    }
    for (size_t i = 0; i < more; ++i) {
      s->table.push_back(free_blocks.back());
      free_blocks.pop_back();
    }
    return KANSO_OK;
  }
  void release(Sequence* s) {
    for (size_t i = s->first_live; i < s->table.size(); ++i) free_blocks.push_back(s->table[i]);
    if (s->slot != NO_SLOT) free_slots.push_back(s->slot);
    *s = Sequence();
  }
  // Gives back the pages that no later token can see.
  void retire(Sequence* s) {
    const uint32_t w = model->max_window();
    if (!w || s->len + 1 <= w) return;
    const uint32_t keep_from = s->len + 1 - w;
    for (; (uint64_t)(s->first_live + 1) * block_size <= keep_from; ++s->first_live) {
      free_blocks.push_back(s->table[s->first_live]);
      s->table[s->first_live] = 0;
    }
  }

  // One model step; the wanted rows' logits are left in model->logits.
  int32_t run(const std::vector<Portion>& ps, const std::vector<uint32_t>& want) {
    tokens.clear();
    query_lens.clear();
    context_lens.clear();
    slots.clear();
    size_t max_blocks = 1;
    for (const Portion& p : ps) {
      const int32_t st = reserve(p.seq, p.n);
      if (st) return st;
      max_blocks = std::max(max_blocks, p.seq->table.size());
    }
    tables.assign(ps.size() * max_blocks, 0);
    for (size_t i = 0; i < ps.size(); ++i) {
      const Portion& p = ps[i];
      tokens.insert(tokens.end(), p.tokens, p.tokens + p.n);
      query_lens.push_back(p.n);
      context_lens.push_back(p.seq->len + p.n);
      slots.push_back(p.seq->slot);
      std::copy(p.seq->table.begin(), p.seq->table.end(), tables.begin() + i * max_blocks);
    }
    StepBatch b;
    b.S = (uint32_t)ps.size();
    b.T = (uint32_t)tokens.size();
    b.max_blocks = (uint32_t)max_blocks;
    b.tokens = tokens.data();
    b.query_lens = query_lens.data();
    b.context_lens = context_lens.data();
    b.tables = tables.data();
    b.state_slots = slots.data();
    b.want = want.data();
    b.n_want = (uint32_t)want.size();
    const int32_t st = run_step(model, kv, b);
    if (st) return st;
    for (const Portion& p : ps) {
      p.seq->len += p.n;
      retire(p.seq);
    }
    return KANSO_OK;
  }
};

extern "C" {

int32_t kanso_cuda_engine_create(kanso_cuda_model* m, uint32_t max_tokens, uint32_t max_seqs,
                                 kanso_cuda_engine** out) {
  if (!m) return fail(nullptr, KANSO_ERR_CONFIG, "engine_create: model is NULL");
  kanso_cuda_ctx* ctx = m->ctx;
  if (!out || !max_tokens || !max_seqs)
    return fail(ctx, KANSO_ERR_CONFIG, "engine_create: every size must be non-zero");
  *out = nullptr;
  auto* e = new kanso_cuda_engine;
  e->model = m;
  e->ctx = ctx;
  e->block_size = m->block_size();
  e->max_seqs = max_seqs;
  // every request may leave its last page partly filled, and its first one partly retired
  e->num_blocks = (max_tokens + e->block_size - 1) / e->block_size + 2 * max_seqs;
  const int32_t st = m->create_pool(e->num_blocks, max_seqs, &e->kv);
  if (st) {
    delete e;
    return st;
  }
  for (uint32_t b = e->num_blocks; b-- > 0;) e->free_blocks.push_back(b);
  for (uint32_t s = max_seqs; s-- > 0;) e->free_slots.push_back(s);
  *out = e;
  return KANSO_OK;
}

int32_t kanso_cuda_engine_destroy(kanso_cuda_engine* e) {
  if (!e) return KANSO_OK;
  cudaDeviceSynchronize();  // the context may already be destroyed
  delete e;
  return KANSO_OK;
}

int32_t kanso_cuda_engine_step(kanso_cuda_engine* e, uint32_t n_entries, const uint64_t* ids,
                               const uint32_t* n_tokens, const uint32_t* tokens,
                               const uint32_t* n_want, const uint32_t* want, float* logits_out) {
  if (!e) return fail(nullptr, KANSO_ERR_CONFIG, "engine_step: engine is NULL");
  kanso_cuda_ctx* ctx = e->ctx;
  if (!n_entries) return KANSO_OK;
  if (!ids || !n_tokens || !tokens || !n_want)
    return fail(ctx, KANSO_ERR_SHAPE, "engine_step: NULL argument");
  // Where an entry's tokens, wants and result rows lie.
  struct Entry {
    Sequence* seq;
    const uint32_t* tokens;
    uint32_t n, done;
    std::vector<std::pair<uint32_t, uint64_t>> want;  // (place, row of the result), by place
    size_t next_want;
  };
  std::vector<Entry> es(n_entries);
  uint64_t tok_at = 0, row_at = 0;
  size_t fresh = 0;
  for (uint32_t i = 0; i < n_entries; ++i) {
    if (!n_tokens[i]) return fail(ctx, KANSO_ERR_SHAPE, "engine_step: an entry without tokens");
    if (n_want[i] && (!want || !logits_out))
      return fail(ctx, KANSO_ERR_SHAPE, "engine_step: NULL argument");
    for (uint32_t k = 0; k < i; ++k)
      if (ids[k] == ids[i])
        return fail(ctx, KANSO_ERR_SHAPE, "engine_step: request %llu twice in a step",
                    (unsigned long long)ids[i]);
    for (uint32_t k = 0; k < n_want[i]; ++k)
      if (want[row_at + k] >= n_tokens[i])
        return fail(ctx, KANSO_ERR_SHAPE, "engine_step: logits of token %u of %u", want[row_at + k],
                    n_tokens[i]);
    fresh += e->live.count(ids[i]) == 0;
    row_at += n_want[i];
  }
  if (e->live.size() + fresh > e->max_seqs)
    return fail(ctx, KANSO_ERR_SHAPE, "engine_step: more than %u live requests", e->max_seqs);
  row_at = 0;
  for (uint32_t i = 0; i < n_entries; ++i) {
    Entry& en = es[i];
    en.seq = &e->live[ids[i]];  // references stay valid while other requests are added
    en.tokens = tokens + tok_at;
    en.n = n_tokens[i];
    en.done = 0;
    en.next_want = 0;
    for (uint32_t k = 0; k < n_want[i]; ++k) en.want.emplace_back(want[row_at + k], row_at + k);
    std::stable_sort(en.want.begin(), en.want.end(),
                     [](const auto& a, const auto& b) { return a.first < b.first; });
    tok_at += n_tokens[i];
    row_at += n_want[i];
  }
  const uint32_t limit = e->model->max_query_len(), vocab = e->model->vocab_size();
  std::vector<Portion> ps;
  std::vector<uint32_t> rows;
  std::vector<uint64_t> dest;
  while (true) {
    ps.clear();
    rows.clear();
    dest.clear();
    uint32_t budget = MAX_STEP_TOKENS, row = 0;
    for (Entry& en : es) {
      uint32_t n = std::min(en.n - en.done, budget);
      if (limit) n = std::min(n, limit);
      if (!n) continue;
      ps.push_back({en.seq, en.tokens + en.done, n});
      for (; en.next_want < en.want.size() && en.want[en.next_want].first < en.done + n;
           ++en.next_want) {
        rows.push_back(row + en.want[en.next_want].first - en.done);
        dest.push_back(en.want[en.next_want].second);
      }
      en.done += n;
      budget -= n;
      row += n;
    }
    if (ps.empty()) break;
    int32_t st = e->run(ps, rows);
    if (st) return st;
    // runs of consecutive result rows go in one copy
    for (size_t i = 0; i < dest.size();) {
      size_t k = i + 1;
      while (k < dest.size() && dest[k] == dest[k - 1] + 1) ++k;
      KANSO_CUDA_TRY(ctx,
                     cudaMemcpyAsync(logits_out + dest[i] * vocab,
                                     e->model->logits + i * vocab, (k - i) * vocab * 4,
                                     cudaMemcpyDeviceToHost, ctx->stream),
                     "d2h");
      i = k;
    }
    if ((st = kanso_cuda_sync(ctx))) return st;
  }
  return KANSO_OK;
}

int32_t kanso_cuda_engine_end(kanso_cuda_engine* e, uint64_t id) {
  if (!e) return fail(nullptr, KANSO_ERR_CONFIG, "engine_end: engine is NULL");
  auto it = e->live.find(id);
  if (it == e->live.end())
    return fail(e->ctx, KANSO_ERR_SHAPE, "engine_end: no request %llu", (unsigned long long)id);
  e->release(&it->second);
  e->live.erase(it);
  return KANSO_OK;
}

uint32_t kanso_cuda_engine_free_blocks(const kanso_cuda_engine* e) {
  return e ? (uint32_t)e->free_blocks.size() : 0;
}

int32_t kanso_cuda_engine_generate(kanso_cuda_engine* e, uint32_t n_prompts,
                                   const uint32_t* prompt_lens, const uint32_t* prompts,
                                   uint32_t max_new, uint32_t max_step_tokens, uint32_t* out) {
  if (!e) return fail(nullptr, KANSO_ERR_CONFIG, "engine_generate: engine is NULL");
  kanso_cuda_ctx* ctx = e->ctx;
  if (!n_prompts || !max_new) return KANSO_OK;
  if (!prompt_lens || !prompts || !out)
    return fail(ctx, KANSO_ERR_SHAPE, "engine_generate: NULL argument");
  const uint32_t step_tokens =
      std::min(max_step_tokens ? max_step_tokens : DEFAULT_STEP_TOKENS, MAX_STEP_TOKENS);
  const uint32_t limit = e->model->max_query_len(), window = e->model->max_window();
  struct Request {
    Sequence seq;
    const uint32_t* prompt = nullptr;
    uint32_t prompt_len = 0, made = 0, pages = 0;
    uint32_t* out = nullptr;
  };
  std::vector<Request> reqs(n_prompts);
  std::deque<uint32_t> waiting;
  std::vector<uint32_t> running;
  const uint32_t capacity = (uint32_t)e->free_blocks.size();
  uint64_t at = 0;
  for (uint32_t i = 0; i < n_prompts; ++i) {
    Request& r = reqs[i];
    r.prompt = prompts + at;
    r.prompt_len = prompt_lens[i];
    r.out = out + (size_t)i * max_new;
    at += prompt_lens[i];
    if (!r.prompt_len) return fail(ctx, KANSO_ERR_SHAPE, "engine_generate: an empty prompt");
    // the most pages the request holds at a time: all of it, or a window and a portion
    uint64_t held = (uint64_t)r.prompt_len + max_new;
    if (window) held = std::min<uint64_t>(held, (uint64_t)window + step_tokens + e->block_size);
    r.pages = (uint32_t)((held + e->block_size - 1) / e->block_size) + 1;
    if (r.pages > capacity)
      return fail(ctx, KANSO_ERR_SHAPE, "engine_generate: request %u needs %u cache pages of %u", i,
                  r.pages, capacity);
    waiting.push_back(i);
  }
  uint32_t promised = 0;
  std::vector<Portion> ps;
  std::vector<uint32_t> want, who, next;
  int32_t st = KANSO_OK;
  while (!st && !(waiting.empty() && running.empty())) {
    while (!waiting.empty() && e->live.size() + running.size() < e->max_seqs &&
           promised + reqs[waiting.front()].pages <= capacity) {
      promised += reqs[waiting.front()].pages;
      running.push_back(waiting.front());
      waiting.pop_front();
    }
    if (running.empty()) {
      st = fail(ctx, KANSO_ERR_SHAPE, "engine_generate: live requests leave no room for another");
      break;
    }
    // decoding requests first, one token each; prompts share what is left of the step
    ps.clear();
    want.clear();
    who.clear();
    uint32_t budget = step_tokens, row = 0;
    for (int prompts_turn = 0; prompts_turn < 2; ++prompts_turn)
      for (uint32_t i : running) {
        Request& r = reqs[i];
        const bool in_prompt = r.seq.len < r.prompt_len;
        if (in_prompt != (prompts_turn == 1) || !budget) continue;
        uint32_t n = in_prompt ? std::min(r.prompt_len - r.seq.len, budget) : 1;
        if (limit) n = std::min(n, limit);
        ps.push_back({&r.seq, in_prompt ? r.prompt + r.seq.len : r.out + (r.made - 1), n});
        if (r.seq.len + n >= r.prompt_len) {
          want.push_back(row + n - 1);
          who.push_back(i);
        }
        row += n;
        budget -= n;
      }
    if ((st = e->run(ps, want))) break;
    if (want.empty()) {
      st = kanso_cuda_sync(ctx);
      continue;
    }
    if (want.size() > e->d_next_cap) {
      if (e->d_next) cudaFree(e->d_next);
      e->d_next = nullptr;
      const cudaError_t ce = cudaMalloc((void**)&e->d_next, want.size() * 4);
      if (ce != cudaSuccess) {
        e->d_next_cap = 0;
        st = cuda_fail(ctx, ce, "engine_generate");
        break;
      }
      e->d_next_cap = want.size();
    }
    next.resize(want.size());
    st = kanso_cuda_greedy_token(ctx, e->model->logits, e->d_next, (int64_t)want.size(),
                                 e->model->vocab_size());
    if (st) break;
    const cudaError_t ce = cudaMemcpyAsync(next.data(), e->d_next, want.size() * 4,
                                           cudaMemcpyDeviceToHost, ctx->stream);
    if (ce != cudaSuccess) {
      st = cuda_fail(ctx, ce, "engine_generate");
      break;
    }
    if ((st = kanso_cuda_sync(ctx))) break;
    for (size_t k = 0; k < who.size(); ++k) {
      Request& r = reqs[who[k]];
      r.out[r.made++] = next[k];
      if (r.made == max_new) {
        e->release(&r.seq);
        promised -= r.pages;
        running.erase(std::find(running.begin(), running.end(), who[k]));
      }
    }
  }
  for (Request& r : reqs) e->release(&r.seq);  // after an error
  return st;
}

}  // extern "C"
