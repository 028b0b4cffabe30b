// What every model shares: the token loop (embed, forward, prefill, pick, generate) and the handling of per-sequence caches —
// the C++ mirror of the model-independent part of crates/det/src/model.rs (Sampling, Model::{set_all_logits, reset, forward,
// logits, pick, prefill, generate}).  A concrete model (qwen35.hpp, hybrid.hpp) supplies its network and its caches; the
// batched decoder (serve.hpp), the graph decoder (graph_decode.hpp) and the C entry points work on this interface.  A model
// talks to a backend only through the op set of backend.hpp.
#pragma once
#include "backend.hpp"
#include "comm.hpp"
#include "hooks.hpp"
#include <functional>
#include <memory>
#include <string>
#include <vector>

namespace det {

struct Sampling {   // model.rs:120-141
    bool greedy = true;
    float inv_temp = 1.0f;
    size_t top_k = 0;
    float top_p = 1.0f;
    uint64_t rng = 0;
};

// Everything one sequence keeps between steps, in every layer (a key/value cache, a recurrent state, ...).  A model makes
// them for as many sequences as a caller holds; exactly one is bound to the model at a time.
struct SeqCache {
    virtual ~SeqCache() = default;
};

// The per-sequence caches / states behind the rows of a batched decode step (serve.hpp): with it the network takes row b
// of the step's activations as the current token of sequence b, at the position pos[b] of that sequence.
struct RowsCtx {
    const std::vector<std::unique_ptr<RowSet>>* sets;   // one per layer
    const Buf<int32_t>* pos;                            // [rows], backend memory
    size_t max_pos;                                     // host bound on the positions
};

// The embedding table in backend memory, for steps whose token comes from the device.
struct EmbedTable {
    const void* table = nullptr;
    int type = 30;   // ggml type: 0 F32, 1 F16, 30 BF16
};

class Model {
  public:
    virtual ~Model() = default;
    Model() = default;
    Model(const Model&) = delete;
    Model& operator=(const Model&) = delete;

    virtual size_t vocab() const = 0;
    virtual size_t hidden() const = 0;
    // Residual rows of `t` tokens into x; "" on success (model.rs:389-413).
    virtual std::string embed_rows(const int32_t* ids, size_t t) = 0;
    // The network over the `t` rows of x: positions pos0 .. pos0 + t of the bound sequence, or one row per sequence with
    // `rows`.  Leaves logits in logits_buf: of the rows named by forward_rows(), of every row when all_logits, else of the last.
    virtual void network(size_t pos0, size_t t, Observer* obs = nullptr, const RowsCtx* rows = nullptr) = 0;

    // ---- caches of further sequences
    virtual std::unique_ptr<SeqCache> new_sequence(size_t ctx) = 0;      // room for ctx positions, cleared
    virtual void swap_sequence(SeqCache& s) = 0;                          // exchanges the bound caches with these
    virtual void clear_sequence(SeqCache& s) = 0;                         // back to position 0
    virtual std::vector<std::unique_ptr<RowSet>> make_rowsets(const std::vector<SeqCache*>& seqs) = 0;   // one per layer
    virtual EmbedTable embed_table() = 0;

    void set_all_logits(bool all);                                   // model.rs:367-375
    void reset();                                                    // model.rs:377-387
    std::string forward(const int32_t* ids, size_t t, Observer* obs = nullptr);            // model.rs:439-465
    // One step whose logits are wanted for the given rows (ascending or not, possibly none), in that order in logits_buf.
    std::string forward_rows(const int32_t* ids, size_t t, const std::vector<int32_t>& want);
    std::vector<float> logits();                                     // model.rs:467-470
    std::string pick(Sampling& s, int32_t& id);                      // model.rs:472-496
    std::string pick_row(const Buf<float>& logits_row, Sampling& s, int32_t& id);   // the same draw on a given logits row
    static uint64_t next_draw(Sampling& s);   // advances the generator once, returns z (model.rs:484-485)
    std::string prefill(const int32_t* ids, size_t n, Observer* obs = nullptr);            // model.rs:498-508
    std::string generate(const int32_t* prompt, size_t n_prompt, size_t n_new, Sampling s,
                         const std::vector<int32_t>& stop, std::vector<int32_t>& out,
                         const std::function<void(int32_t)>& on_token = nullptr, Observer* obs = nullptr);   // model.rs:510-547

    Backend* backend = nullptr;
    size_t max_ctx = 0, max_batch = 0, pos = 0;
    bool all_logits = false;
    Buf<float> x;            // residual rows [max_batch][hidden]
    Buf<float> logits_buf;   // [vocab], or one row per requested position

  protected:
    virtual void clear_bound() = 0;                 // the bound sequence back to its start
    virtual void logits_resized(size_t) {}
    const std::vector<int32_t>* head_rows_ = nullptr;   // set while forward_rows() runs
};

}  // namespace det
