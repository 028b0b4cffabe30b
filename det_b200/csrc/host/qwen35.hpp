// The Qwen3.5 model (Gated DeltaNet + gated attention over quantized linears) — the C++ mirror of crates/det/src/model.rs
// (Proj, Attn, Gdn, Layer, Work, Model::{load, embed_rows, project}) and of the network's op sequence
// crates/det/src/qwen35.rs:8-172.  The same driver runs the CUDA backend and, in tests, the CPU reference backend.
#pragma once
#include "gguf.hpp"
#include "model.hpp"
#include "synth.hpp"

namespace det {

constexpr float DEFAULT_V_SCALE = 1.0f / 1024.0f;   // model.rs:47

struct Proj {   // model.rs:51-53
    std::vector<std::unique_ptr<Linear>> lins;
};
struct Attn {   // model.rs:55-63
    Proj qkv, o;
    Buf<float> q_norm, k_norm, v_scale, v_inv_scale;
    KvCache kv;
};
struct Gdn {   // model.rs:65-74
    Proj qkvz, ab, out;
    Buf<float> conv, a, dt_bias, norm;
    GdnState state;
};
struct Layer {   // model.rs:81-87
    Buf<float> attn_norm, ffn_norm;
    Proj gu, down;
    bool is_attn = false;
    Attn attn;
    Gdn gdn;
};
struct Work {   // model.rs:89-118
    Buf<int8_t> xq;
    Buf<float> sx;
    Buf<uint16_t> mx;
    Buf<float> qg, k, v, o;
    Buf<int8_t> oq;
    Buf<float> so;
    Buf<uint16_t> mo;
    Buf<float> qkv, z, a, b, on;
    Buf<int8_t> onq;
    Buf<float> son;
    Buf<uint16_t> mon;
    Buf<float> g, u;
    Buf<int8_t> hq;
    Buf<float> sh;
    Buf<uint16_t> mh;
    Buf<float> gin, gout;   // GDN mixer export (model.rs:343-344); sized on the first observed step that asks for them
};
// One sequence's caches, in layer order: a KvCache per attention layer, a GdnState per Gated DeltaNet layer.
struct Qwen35Cache : SeqCache {
    std::vector<KvCache> kv;
    std::vector<GdnState> st;
};

class Qwen35Model : public Model {
  public:
    // A seeded random-init model of shape `cfg` (the stand-in for Model::load on a converted checkpoint).
    // `comm` (optional) makes this the shard of rank comm->rank in a tensor-parallel group of comm->size: linears are
    // cut by output rows, attention by q heads, Gated DeltaNet by k heads, the FFN by 128-column groups, the head by
    // vocabulary rows; the residual stream and the norms stay replicated (see network_tp in qwen35.cpp).
    static std::unique_ptr<Qwen35Model> load_synthetic(const Config& cfg, uint64_t seed, Backend* backend, size_t max_ctx,
                                                       size_t max_batch, Comm* comm = nullptr);

    // Model::load (model.rs:164-365): a det GGUF written by `det convert` (or write_synthetic_gguf).  Null and a message in
    // `err` when the file is unreadable, not a qwen35 det file, holds a non-finite value, or lacks a tensor.
    static std::unique_ptr<Qwen35Model> load(const std::string& path, Backend* backend, size_t max_ctx, size_t max_batch,
                                             std::string& err);

    size_t vocab() const override { return cfg.vocab; }
    size_t hidden() const override { return cfg.hidden; }
    std::string embed_rows(const int32_t* ids, size_t t) override;   // model.rs:389-413
    void network(size_t pos0, size_t t, Observer* obs = nullptr, const RowsCtx* rows = nullptr) override;   // qwen35.rs:8-172
    std::unique_ptr<SeqCache> new_sequence(size_t ctx) override;
    void swap_sequence(SeqCache& s) override;
    void clear_sequence(SeqCache& s) override;
    std::vector<std::unique_ptr<RowSet>> make_rowsets(const std::vector<SeqCache*>& seqs) override;
    EmbedTable embed_table() override;
    void project(const Proj& p, const Buf<int8_t>& xq, const Buf<float>& sx, const Buf<uint16_t>& mx, size_t t,
                 const std::vector<const Buf<float>*>& dsts);        // model.rs:415-437

    Config cfg;
    uint64_t seed = 0;
    std::shared_ptr<Gguf> gguf;   // the mapped file of a loaded model (null for a synthetic one); owns the embedding rows
    GgufTensor embed;             // token_embd.weight of `gguf`
    bool calibrated = false;      // the file carries value scales other than the default (model.rs:236-244)
    Buf<float> final_norm, rope_cos, rope_sin;
    Proj lm_head;
    std::vector<Layer> layers;
    Work w;

    // ---- tensor parallel state (comm == nullptr: none of it is used)
    Comm* comm = nullptr;
    struct Tp {
        size_t heads = 0, kv = 0;        // local q heads / kv heads of an attention layer
        size_t k_heads = 0, v_heads = 0; // local GDN heads
        size_t ffn = 0, hid = 0, voc = 0;   // local FFN columns, hidden rows, vocabulary rows
        Buf<float> mix_full;   // [mb][n_h*hd] gathered mixer output
        Buf<float> h_l, h_full;      // SwiGLU product, local and gathered
        Buf<float> y_l, y_full;      // projection back to hidden, local rows and gathered
        Buf<float> logits_l;
        Buf<float> tmp;              // all-gather scratch
        Buf<float> x_alt;            // second copy of the residual stream (an exchange fused into a GEMV stores the sums here)
    } tp;

  protected:
    void clear_bound() override;
    void logits_resized(size_t n) override;

  private:
    void network_tp(size_t pos0, size_t t, const RowsCtx* rows);
    Buf<uint8_t> embed_dev_;   // device copy of the embedding table, made by the first embed_table()
};

}  // namespace det
