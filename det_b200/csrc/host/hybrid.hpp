// Decoder models built from a list of layers, each with a mixer of its own kind and sizes and an optional feed-forward, over
// bfloat16 linears and an fp32 residual stream.  Two designs of the registry are built so.
//
// "Fazilorn" (parallel layers):
//   x <- x + (mixer(h) + ff(h)), h = RMSnorm(x): both sublayers read one norm, so a layer is two products around the mixer —
//     every projection of h (the feed-forward's gate and up included, their SwiGLU in the epilogue) as one launch, and
//     [W_o | W_down] over the concatenated [mixer output | SwiGLU product] as one accumulating launch.
//   mixers: gated linear attention ("gla"), RWKV-style time mixing ("wkv") — one recurrence with different decays, token
//     shift and bonus — and latent attention with a sliding window, a sink and an output gate ("latent_attention").
//   a layer may use the tensors of an earlier one (weights_of) with a cache or state of its own.
//
// "Dopipel" (serial layers):
//   x <- x + scale1 * RMSnorm(mixer(h + conv(h))), h = RMSnorm(x), conv a short causal convolution per channel;
//   x <- x + scale2 * RMSnorm(ff(RMSnorm(x))): a norm on both ends of a sublayer.  What lies between two sublayers (result norm,
//     layer scale, residual add, next norm, convolution) is one launch, det_f_seam; a sublayer is a product, its core, a product.
//   mixers: attention over grouped key/value heads with rotated values and a gate per head, and a minimal gated recurrence.
//   feed-forward: pairs behind a relu, or a mixture of experts with identity experts and a gated shared expert.
//   a range of layers may run several times in a row (loop) with a cache or state per pass; ahead of each pass the residual row is
//     mixed with the token's embedding row and a vector of the pass is added.
#pragma once
#include "json.hpp"
#include "model.hpp"
#include <array>

namespace det {

enum class MixerKind { Gla, Wkv, Latent, Attention, MinGru };

struct MixerSpec {
    MixerKind kind = MixerKind::Gla;
    size_t heads = 0, dim = 0, vdim = 0;
    float tau = 1.0f;                                     // gla
    size_t q_rank = 0, kv_rank = 0, rot_dim = 0, rot_dims = 0;   // latent attention
    double rot_base = 10000.0;
    size_t window = 0;                                    // 0: every earlier token
    float scale = 1.0f;
    size_t kv_heads = 0;                                  // attention
    size_t width = 0;                                     // mingru
    size_t width_out() const { return kind == MixerKind::MinGru ? width : heads * vdim; }     // what W_o reads
};
struct MoeSpec {
    size_t experts = 0;         // 0: no mixture
    size_t identity = 0, top = 0, ff = 0;
    size_t shared = 0;          // inner size of the shared expert, 0: none
    size_t outputs() const { return experts + identity; }
};
struct LayerSpec {
    MixerSpec mixer;
    size_t ff = 0;              // dense feed-forward, 0: none
    MoeSpec moe;
    size_t weights = 0;         // the layer whose tensors this one uses (itself, mostly)
};
// One run of a layer; each has a cache or state of its own.
struct LayerRun {
    size_t layer = 0;
    int pass = -1;              // the pass of the loop that begins here, or -1
};
struct HybridConfig {
    size_t vocab = 0, width = 0;
    float eps = 1e-5f;
    float softcap = 0.0f;       // 0: none
    bool serial = false;        // layers of the serial form
    size_t taps = 0;            // of the convolution ahead of a serial layer's mixer, 0: none
    size_t passes = 0;          // of the loop, 0: none
    std::vector<LayerSpec> layers;
    std::vector<LayerRun> runs;
    // Throws std::runtime_error naming the layer and the key on anything missing, unknown or inconsistent.
    static HybridConfig from_json(const Json& j);
};

// Where a model's tensors come from: a file, or a seeded generator (benchmarks).
struct TensorSource {
    virtual ~TensorSource() = default;
    // rows x cols bfloat16 values of a tensor, row-major, into `out`; throws when it is absent or has another shape
    virtual void matrix(const std::string& name, size_t rows, size_t cols, uint16_t* out) = 0;
    virtual std::vector<float> vector(const std::string& name, size_t n) = 0;
    virtual size_t rows_of(const std::string& name, size_t cols) = 0;   // leading size of a matrix whose width is known
    // Fills a device matrix in place instead (false: not supported).
    virtual bool on_device(const std::string&, size_t, size_t, uint16_t*) { return false; }
};

struct HybridWeights {
    Buf<float> norm1;
    FLinear in;                         // every projection of the normalised row; gate / up rows interleaved at the end
    size_t plain = 0;                   // rows of `in` before the gate / up pairs
    size_t off[5] = {0, 0, 0, 0, 0};    // columns of the parts: q k v g a1 | r k v g w1 | dq dkv g | q k v g | z x g
    FLinear out;                        // [W_o | zeros to a multiple of 8 | W_down]
    size_t out_ff = 0;                  // first column of the SwiGLU product
    // recurrences
    Buf<float> mu;                      // [5][width] token-shift mixes (wkv)
    FLinear decay;                      // second half of the low-rank decay projection
    size_t rank = 0;
    Buf<float> decay_bias, bonus, head_norm;
    // latent attention
    Buf<float> dq_norm, dkv_norm, sink;
    FLinear uq, ukv;
    // serial layers
    Buf<float> norm1b, norm2, norm2b, scale1, scale2;
    Buf<float> conv;                    // [taps][width]
    Buf<float> in_bias, out_bias;
    FLinear ff_in;                      // gate / up pairs, or [router | shared gate | shared first half]
    size_t ff_plain = 0;                // rows of ff_in before those of a first half
    FLinear ff_out;                     // second half, of the shared expert in a mixture
    FLinear up, down;                   // stacks of the experts' halves
    Buf<float> correction;
};
struct HybridCache : SeqCache {
    std::vector<FloatState> layers;     // one per layer run
};

class HybridModel : public Model {
  public:
    static std::unique_ptr<HybridModel> load(const HybridConfig& cfg, TensorSource& src, Backend* backend, size_t max_ctx,
                                             size_t max_batch, Dtype dtype);
    // config.json + model.safetensors of a folder
    static std::unique_ptr<HybridModel> load_dir(const std::string& dir, const Json& config, Backend* backend, size_t max_ctx,
                                                 size_t max_batch, Dtype dtype);
    // seeded random weights (std 0.02, unit norms)
    static std::unique_ptr<HybridModel> load_synthetic(const Json& config, uint64_t seed, Backend* backend, size_t max_ctx,
                                                       size_t max_batch, Dtype dtype);

    size_t vocab() const override { return cfg.vocab; }
    size_t hidden() const override { return cfg.width; }
    std::string embed_rows(const int32_t* ids, size_t t) override;
    void network(size_t pos0, size_t t, Observer* obs = nullptr, const RowsCtx* rows = nullptr) override;
    std::unique_ptr<SeqCache> new_sequence(size_t ctx) override;
    void swap_sequence(SeqCache& s) override;
    void clear_sequence(SeqCache& s) override;
    std::vector<std::unique_ptr<RowSet>> make_rowsets(const std::vector<SeqCache*>& seqs) override;
    EmbedTable embed_table() override { return EmbedTable{embed_.ptr(), 30}; }
    size_t weight_bytes() const;   // read by one decoded token: linears once per layer run, head once

    HybridConfig cfg;
    Dtype dtype = Dtype::BF16;

  protected:
    void clear_bound() override { clear_sequence(bound_); }

  private:
    struct Rope {
        double base;
        size_t dims;
        Buf<float> cos, sin;   // [max_ctx][dims / 2]
    };
    void mixer_recurrent(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq);
    void mixer_latent(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq, size_t cap, size_t max_pos);
    void mixer_attention(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq, size_t cap, size_t max_pos);
    void mixer_mingru(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq);
    void parallel_layer(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq, size_t cap, size_t max_pos);
    void serial_mixer(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq, size_t cap, size_t max_pos);
    void serial_ff(const LayerSpec& l, const HybridWeights& w, size_t t);
    det_fseam_op seam(size_t t) const;
    void pack_rows(size_t t, size_t col);
    void loop_entry(size_t t, int pass);
    void add_rope(double base, size_t dims);
    void run_in(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq);
    void head(size_t t);
    const Rope& rope(double base, size_t dims) const;

    Buf<uint16_t> embed_;
    std::vector<std::shared_ptr<HybridWeights>> weights_;   // one per layer; shared by layers that share tensors
    Buf<float> final_norm_;
    FLinear head_lin_;
    std::vector<Rope> ropes_;
    HybridCache bound_;
    // activations of one step (max_batch rows)
    Buf<uint8_t> in_, cat_, cq_;
    Buf<float> y_, q_;
    Buf<int32_t> ids_, rows_;
    size_t ld_in_ = 0, ld_cq_ = 0;
    // serial layers: a sublayer's result, reciprocal norms, [residual | embedding] rows ahead of a pass
    Buf<float> res_, rstd_;
    Buf<uint8_t> pair_;
    FLinear loop_lin_;
    Buf<float> loop_step_;              // [passes][width]
    size_t ld_pair_ = 0;
};

}  // namespace det
