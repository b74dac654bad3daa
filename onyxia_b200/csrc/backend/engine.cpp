// Page and slot management, the batch step, the continuous-batching scheduler, and their C entry points.
#include "engine.hpp"

#include <algorithm>
#include <cstring>

#include "../ir/module_api.hpp"
#include "capi_types.hpp"

namespace oxrt {

using namespace ox;

namespace {

bool starts_with(const std::string& s, const char* prefix) { return s.rfind(prefix, 0) == 0; }

// splitmix64 (Steele, Lea, Flood: "Fast splittable pseudorandom number generators"): one uniform in [0, 1) per draw
float next_uniform(uint64_t& state) {
    uint64_t z = (state += 0x9E3779B97F4A7C15ull);
    z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
    z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
    z ^= z >> 31;
    return (float)(z >> 40) * (1.f / 16777216.f);
}

}  // namespace

bool Engine::serves(const Module& m) {
    for (auto& in : m.inputs)
        if (in.first == "seq_info") return true;
    return false;
}

Engine::Engine(Session& s, int64_t max_tokens, int32_t max_seqs) : s_(s), max_seqs_(max_seqs) {
    const Module& m = s.module();
    if (!serves(m)) fail(ErrKind::Binding, "the module has no 'seq_info' input: it does not run ragged batches");
    if (max_tokens <= 0 || max_seqs <= 0) fail(ErrKind::Shape, "an engine needs room for at least one token and one sequence");
    const auto& outs = s.output_names();
    for (size_t o = 0; o < outs.size(); o++)
        if (outs[o] == "logits") logits_out_ = (int)o;
    if (logits_out_ < 0) fail(ErrKind::Binding, "output 'logits' missing");
    const TensorType& lt = m.values[m.outputs[(size_t)logits_out_].second].ty;
    if (lt.dtype != DType::F32 || lt.shape.size() != 2 || !lt.shape[1].as_const()) fail(ErrKind::DType, "output 'logits' must be F32 [num_logits, vocab]");
    vocab_ = (int64_t)*lt.shape[1].as_const();

    for (auto& in : m.inputs) {
        names_.push_back(in.first);
        if (!starts_with(in.first, "pages.") || page_) continue;
        const TensorType& t = m.values[in.second].ty;
        // [num_pages, …, page, …]: key pools carry the page on axis 2, per-token scalars on axis 1
        const size_t axis = t.shape.size() == 2 ? 1 : 2;
        if (t.shape.size() < 2 || !t.shape[axis].as_const()) fail(ErrKind::Shape, "input '" + in.first + "' has no constant page axis");
        page_ = (int64_t)*t.shape[axis].as_const();
    }
    if (!page_) page_ = 64;  // a module without attention keeps no pages; lengths are still counted in them
    n_pages_ = pages_for(max_tokens);
    Bindings b;
    auto bind = [&](const char* name, uint64_t v) {
        if (auto id = m.symbols.get(name)) b.bind(*id, v);
    };
    bind("num_pages", (uint64_t)n_pages_);
    bind("num_slots", (uint64_t)max_seqs);
    state_.resize(names_.size());
    updated_.assign(names_.size(), -1);
    for (size_t i = 0; i < names_.size(); i++) {
        if (!starts_with(names_[i], "pages.") && !starts_with(names_[i], "slots.")) continue;
        const TensorType& t = m.values[m.inputs[i].second].ty;
        std::vector<int64_t> shape;
        for (auto& d : t.shape) shape.push_back((int64_t)d.eval(b));
        state_[i] = s.zeros(t.dtype, shape);
        for (size_t o = 0; o < outs.size(); o++)
            if (outs[o] == "updated." + names_[i]) updated_[i] = (int)o;
        if (updated_[i] < 0) fail(ErrKind::Binding, "output 'updated." + names_[i] + "' missing");
    }
    for (int64_t i = n_pages_; i-- > 0;) free_pages_.push_back((int32_t)i);
    for (int32_t i = max_seqs; i-- > 0;) free_slots_.push_back(i);
}

int64_t Engine::length(int64_t id) const {
    auto it = seqs_.find(id);
    return it == seqs_.end() ? 0 : it->second.past;
}

void Engine::release(int64_t id) {
    auto it = seqs_.find(id);
    if (it == seqs_.end()) fail(ErrKind::Binding, "no live sequence with id " + std::to_string(id));
    // the next owner of these pages and this slot runs behind everything enqueued so far
    for (size_t i = it->second.pages.size(); i-- > 0;) free_pages_.push_back(it->second.pages[i]);
    free_slots_.push_back(it->second.slot);
    seqs_.erase(it);
}

DTensor Engine::forward(const std::vector<Entry>& entries, const DTensor* ids_dev) {
    if (entries.empty()) fail(ErrKind::Shape, "a step needs at least one entry");
    // what the step needs, before anything is taken
    int64_t new_pages = 0, new_slots = 0, rows = 0;
    for (size_t i = 0; i < entries.size(); i++) {
        const Entry& e = entries[i];
        if (e.n_tokens <= 0) fail(ErrKind::Shape, "an entry brings at least one token");
        for (size_t j = 0; j < i; j++)
            if (entries[j].id == e.id) fail(ErrKind::Binding, "sequence " + std::to_string(e.id) + " appears twice in one step");
        for (int32_t w = 0; w < e.n_want; w++)
            if (e.want[w] < 0 || e.want[w] >= e.n_tokens) fail(ErrKind::Shape, "a wanted place lies outside the entry's tokens");
        auto it = seqs_.find(e.id);
        const int64_t past = it == seqs_.end() ? 0 : it->second.past, have = it == seqs_.end() ? 0 : (int64_t)it->second.pages.size();
        if (past + e.n_tokens > INT32_MAX / 2) fail(ErrKind::Shape, "sequence too long");
        new_pages += std::max<int64_t>(0, pages_for(past + e.n_tokens) - have);
        new_slots += it == seqs_.end();
        rows += e.n_tokens;
    }
    if (new_slots > (int64_t)free_slots_.size()) fail(ErrKind::Runtime, "no free slot for a new sequence");
    if (new_pages > (int64_t)free_pages_.size())
        fail(ErrKind::Runtime, "out of cache pages: " + std::to_string(new_pages) + " needed, " + std::to_string(free_pages_.size()) + " free");

    std::vector<int64_t> ids, want;
    std::vector<int32_t> info;
    size_t widest = 1;
    int64_t row = 0;
    for (auto& e : entries) {
        auto it = seqs_.find(e.id);
        if (it == seqs_.end()) {
            it = seqs_.emplace(e.id, Seq{}).first;
            it->second.slot = free_slots_.back();
            free_slots_.pop_back();
        }
        Seq& q = it->second;
        while ((int64_t)q.pages.size() < pages_for(q.past + e.n_tokens)) {
            q.pages.push_back(free_pages_.back());
            free_pages_.pop_back();
        }
        widest = std::max(widest, q.pages.size());
        info.insert(info.end(), {(int32_t)row, e.n_tokens, (int32_t)q.past, q.slot});
        if (!ids_dev) ids.insert(ids.end(), e.tokens, e.tokens + e.n_tokens);
        for (int32_t w = 0; w < e.n_want; w++) want.push_back(row + e.want[w]);
        row += e.n_tokens;
    }
    if (want.empty()) want.push_back(rows - 1);
    // four table widths per power of two: a plan (and its graph) serves a sequence while it grows, and a launch that is
    // sized by the width is not far off
    size_t width = 4;
    for (size_t quarter = 1; width < widest; width += quarter)
        if (width == 8 * quarter) quarter *= 2;
    std::vector<int32_t> table(entries.size() * width, 0);
    for (size_t i = 0; i < entries.size(); i++) {
        const Seq& q = seqs_[entries[i].id];
        std::copy(q.pages.begin(), q.pages.end(), table.begin() + (long)(i * width));
    }
    const int64_t R = (int64_t)entries.size();
    std::vector<std::pair<std::string, DTensor>> feed;
    feed.reserve(names_.size());
    for (size_t i = 0; i < names_.size(); i++) {
        const std::string& n = names_[i];
        DTensor t;
        if (n == "input_ids") t = ids_dev ? *ids_dev : s_.upload(DType::I64, {rows}, ids.data(), ids.size() * 8);
        else if (n == "seq_info") t = s_.upload(DType::I32, {R, 4}, info.data(), info.size() * 4);
        else if (n == "page_table") t = s_.upload(DType::I32, {R, (int64_t)width}, table.data(), table.size() * 4);
        else if (n == "logit_rows") t = s_.upload(DType::I64, {(int64_t)want.size()}, want.data(), want.size() * 8);
        else if (state_[i].buf) t = state_[i];
        else fail(ErrKind::Binding, "input '" + n + "' is not one the engine can fill");
        feed.emplace_back(n, std::move(t));
    }
    auto outs = s_.run(feed);
    for (size_t i = 0; i < names_.size(); i++)
        if (updated_[i] >= 0) state_[i] = outs[(size_t)updated_[i]].second;
    for (auto& e : entries) seqs_[e.id].past += e.n_tokens;
    return outs[(size_t)logits_out_].second;
}

// ───────────────────────────── scheduling ───────────────────────────────
int64_t Engine::submit(std::vector<int64_t> prompt, int32_t max_new, int64_t eos, const Sampling& sampling) {
    if (prompt.empty()) fail(ErrKind::Shape, "Cannot prefill with empty input_ids");
    if (max_new <= 0) fail(ErrKind::Shape, "a request generates at least one token");
    Request r;
    r.id = next_request_++;
    r.pages = pages_for((int64_t)prompt.size() + max_new - 1);  // the last token is never run
    if (r.pages > n_pages_) fail(ErrKind::Shape, "the request needs " + std::to_string(r.pages) + " pages, the engine has " + std::to_string(n_pages_));
    r.prompt = std::move(prompt);
    r.left = max_new;
    r.eos = eos;
    r.sampling = sampling;
    r.rng = sampling.seed;
    waiting_.push_back(std::move(r));
    return waiting_.back().id;
}

void Engine::cancel(int64_t request) {
    for (auto it = waiting_.begin(); it != waiting_.end(); ++it)
        if (it->id == request) {
            waiting_.erase(it);
            return;
        }
    for (auto it = running_.begin(); it != running_.end(); ++it)
        if (it->id == request) {
            reserved_ -= it->pages;
            if (seqs_.count(request)) release(request);
            running_.erase(it);
            return;
        }
}

std::vector<int64_t> Engine::sample(const DTensor& logits, const std::vector<Request*>& rows) {
    std::vector<int64_t> tokens(rows.size());
    const bool greedy = std::all_of(rows.begin(), rows.end(), [](Request* r) { return r->sampling.temperature < 1e-6f; });
    if (greedy) {
        s_.download(s_.argmax_last(logits), tokens.data(), tokens.size() * 8, nullptr);
        return tokens;
    }
    std::vector<DTensor> drawn;
    for (size_t i = 0; i < rows.size(); i++) {
        DTensor one = logits;
        one.shape = {1, vocab_};
        one.offset += i * (size_t)vocab_ * 4;
        const Sampling& p = rows[i]->sampling;
        const float u = next_uniform(rows[i]->rng);
        drawn.push_back(s_.sample_last(one, p.temperature, p.top_k, p.top_p, &u, 1));
    }
    for (size_t i = 0; i < rows.size(); i++) s_.download(drawn[i], &tokens[i], 8, nullptr);
    return tokens;
}

std::vector<Engine::Token> Engine::step(int32_t token_budget) {
    // admission: a request enters when a slot is free and the pages of its whole life are
    while (!waiting_.empty() && (int64_t)running_.size() < max_seqs_ && reserved_ + waiting_.front().pages <= n_pages_) {
        reserved_ += waiting_.front().pages;
        running_.push_back(std::move(waiting_.front()));
        waiting_.pop_front();
    }
    std::vector<Entry> entries;
    std::vector<Request*> sampled;
    std::vector<std::pair<Request*, int32_t>> portions;
    static const int32_t first_place = 0;
    int64_t budget = std::max<int64_t>(token_budget, 1);
    for (auto& r : running_)  // decoding requests first
        if (r.fed == r.prompt.size() && budget > 0) {
            entries.push_back(Entry{r.id, &r.last, 1, &first_place, 1});
            sampled.push_back(&r);
            budget--;
        }
    std::vector<int32_t> last_place(running_.size());
    size_t k = 0;
    for (auto& r : running_)
        if (r.fed < r.prompt.size() && budget > 0) {
            const int32_t n = (int32_t)std::min<int64_t>(budget, (int64_t)(r.prompt.size() - r.fed));
            const bool done = r.fed + (size_t)n == r.prompt.size();
            last_place[k] = n - 1;
            entries.push_back(Entry{r.id, r.prompt.data() + r.fed, n, &last_place[k], done ? 1 : 0});
            k++;
            if (done) sampled.push_back(&r);
            portions.emplace_back(&r, n);
            budget -= n;
        }
    std::vector<Token> out;
    if (entries.empty()) return out;
    const DTensor logits = forward(entries);
    for (auto& pr : portions) pr.first->fed += (size_t)pr.second;
    if (sampled.empty()) return out;
    const std::vector<int64_t> tokens = sample(logits, sampled);
    for (size_t i = 0; i < sampled.size(); i++) {
        Request& r = *sampled[i];
        r.last = tokens[i];
        r.left--;
        out.push_back(Token{r.id, tokens[i], r.left == 0 || tokens[i] == r.eos});
    }
    for (auto& t : out)
        if (t.finished) cancel(t.request);
    return out;
}

}  // namespace oxrt

// ───────────────────────────── C entry points ───────────────────────────
using namespace ox;

struct ox_engine {
    std::unique_ptr<oxrt::Engine> e;
};

#define OX_TRY try {
#define OX_CATCH                                                                          \
    }                                                                                     \
    catch (const ox::Error& e) { return (ox_status)ox::set_error(e); }                    \
    catch (const std::exception& e) { return (ox_status)ox::set_error(ErrKind::Runtime, e.what()); }

extern "C" {

ox_status ox_engine_create(ox_session* session, int64_t max_tokens, int32_t max_seqs, ox_engine** out) {
    OX_TRY
    auto h = std::make_unique<ox_engine>();
    h->e = std::make_unique<oxrt::Engine>(*session->s, max_tokens, max_seqs);
    *out = h.release();
    return OX_OK;
    OX_CATCH
}

void ox_engine_free(ox_engine* e) { delete e; }

ox_status ox_engine_forward(ox_engine* h, const ox_engine_entry* entries, int32_t n_entries, float* logits, size_t logits_cap) {
    OX_TRY
    std::vector<oxrt::Engine::Entry> es;
    size_t wanted = 0;
    for (int32_t i = 0; i < n_entries; i++) {
        es.push_back({entries[i].id, entries[i].tokens, entries[i].n_tokens, entries[i].want, entries[i].n_want});
        wanted += (size_t)std::max(entries[i].n_want, 0);
    }
    if (logits && logits_cap < wanted * (size_t)h->e->vocab()) fail(ErrKind::Shape, "logits buffer too small");
    const oxrt::DTensor t = h->e->forward(es);
    if (logits && wanted) h->e->session().download(t, logits, logits_cap * 4, nullptr);
    return OX_OK;
    OX_CATCH
}

ox_status ox_engine_release(ox_engine* h, int64_t id) {
    OX_TRY
    h->e->release(id);
    return OX_OK;
    OX_CATCH
}

ox_status ox_engine_submit(ox_engine* h, const int64_t* prompt, int32_t n_prompt, int32_t max_new, int64_t eos, float temperature, int64_t top_k,
                           float top_p, uint64_t seed, int64_t* request) {
    OX_TRY
    oxrt::Engine::Sampling s;
    s.temperature = temperature;
    s.top_k = top_k;
    s.top_p = top_p;
    s.seed = seed;
    *request = h->e->submit(std::vector<int64_t>(prompt, prompt + std::max(n_prompt, 0)), max_new, eos, s);
    return OX_OK;
    OX_CATCH
}

ox_status ox_engine_step(ox_engine* h, int32_t token_budget, ox_engine_token* tokens, int32_t cap, int32_t* n_tokens) {
    OX_TRY
    if ((int64_t)cap < h->e->running() + h->e->waiting()) fail(ErrKind::Shape, "room for one token per submitted request is needed");
    const auto got = h->e->step(token_budget);
    for (size_t i = 0; i < got.size(); i++) tokens[i] = ox_engine_token{got[i].request, got[i].token, got[i].finished ? 1 : 0};
    *n_tokens = (int32_t)got.size();
    return OX_OK;
    OX_CATCH
}

ox_status ox_engine_cancel(ox_engine* h, int64_t request) {
    OX_TRY
    h->e->cancel(request);
    return OX_OK;
    OX_CATCH
}

void ox_engine_stats(const ox_engine* h, int64_t out[7]) {
    const oxrt::Engine& e = *h->e;
    const int64_t v[7] = {e.page_size(), e.free_pages(), e.free_slots(), e.live(), e.waiting(), e.running(), e.vocab()};
    std::memcpy(out, v, sizeof(v));
}

}  // extern "C"
