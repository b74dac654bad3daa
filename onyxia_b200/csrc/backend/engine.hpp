// Batched serving over a module with paged caches and per-sequence state.
//
// Such a module takes, beside `input_ids` I64 [num_tokens]:
//   seq_info    I32 [num_seqs, 4]: first row, new tokens, tokens before them, slot — the batch is the concatenation
//               of its sequences' new tokens
//   page_table  I32 [num_seqs, table_width]
//   logit_rows  I64 [num_logits]: the batch rows whose logits are wanted
//   pages.*     pools whose first axis is num_pages; axis `page_size` of every one is the same
//   slots.*     per-sequence state whose first axis is num_slots
// and returns `logits` F32 [num_logits, vocab] and every pages.* / slots.* tensor, updated in place, under the name
// "updated.<input>".
#pragma once
#include <deque>

#include "session.hpp"

namespace oxrt {

class Engine {
public:
    struct Entry {
        int64_t id;
        const int64_t* tokens;  // null: `ids_dev` of forward() holds the batch's ids
        int32_t n_tokens;
        const int32_t* want;    // places among the new tokens
        int32_t n_want;
    };
    struct Sampling {
        float temperature = 0.f, top_p = 1.f;
        int64_t top_k = 0;
        uint64_t seed = 0;
    };
    struct Token {
        int64_t request, token;
        bool finished;
    };

    // Room for `max_tokens` tokens (each sequence's count rounded up to whole pages) and `max_seqs` sequences.
    Engine(Session& s, int64_t max_tokens, int32_t max_seqs);
    static bool serves(const Module& m);

    // One step of a batch. A sequence is admitted at its first entry. Returns the wanted rows' logits in entry order
    // (one row that nobody asked for when nothing is wanted). Nothing changes when it fails before the launch.
    DTensor forward(const std::vector<Entry>& entries, const DTensor* ids_dev = nullptr);
    void release(int64_t id);
    int64_t length(int64_t id) const;

    // Continuous batching: every step decodes one token of each running request and spends what is left of the
    // token budget on portions of prompts.
    int64_t submit(std::vector<int64_t> prompt, int32_t max_new, int64_t eos, const Sampling& sampling);
    std::vector<Token> step(int32_t token_budget);
    void cancel(int64_t request);

    Session& session() { return s_; }
    int64_t page_size() const { return page_; }
    int64_t free_pages() const { return (int64_t)free_pages_.size(); }
    int64_t free_slots() const { return (int64_t)free_slots_.size(); }
    int64_t live() const { return (int64_t)seqs_.size(); }
    int64_t waiting() const { return (int64_t)waiting_.size(); }
    int64_t running() const { return (int64_t)running_.size(); }
    int64_t vocab() const { return vocab_; }

private:
    struct Seq {
        int64_t past = 0;
        int32_t slot = 0;
        std::vector<int32_t> pages;
    };
    struct Request {
        int64_t id;
        std::vector<int64_t> prompt;
        size_t fed = 0;       // prompt tokens already run
        int64_t last = -1;    // the token to run next once the prompt is done
        int32_t left;         // tokens still to generate
        int64_t eos;
        Sampling sampling;
        uint64_t rng;
        int64_t pages;        // reserved for its whole life
    };
    int64_t pages_for(int64_t tokens) const { return (tokens + page_ - 1) / page_; }
    std::vector<int64_t> sample(const DTensor& logits, const std::vector<Request*>& rows);

    Session& s_;
    int64_t page_ = 0, n_pages_ = 0, vocab_ = 0;
    std::vector<std::string> names_;   // module inputs, signature order
    std::vector<DTensor> state_;       // per input: the pool or slot tensor
    std::vector<int> updated_;         // per input: the output that hands it back, or −1
    int logits_out_ = -1;
    std::vector<int32_t> free_pages_, free_slots_;
    std::unordered_map<int64_t, Seq> seqs_;
    std::deque<Request> waiting_;
    std::vector<Request> running_;
    int64_t next_request_ = (int64_t)1 << 40,  // apart from the ids a caller of forward() picks
             reserved_ = 0, max_seqs_ = 0;
};

}  // namespace oxrt
