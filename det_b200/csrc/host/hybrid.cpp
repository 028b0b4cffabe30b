#include "hybrid.hpp"
#include "safetensors.hpp"
#include "synth.hpp"
#include <algorithm>
#include <cmath>
#include <cstring>
#include <stdexcept>

namespace det {

namespace {
size_t round8(size_t n) { return (n + 7) & ~(size_t)7; }
[[noreturn]] void bad(const std::string& what) { throw std::runtime_error(what); }
// A product of t rows whose outputs all are plain; input and output still to be named.
det_fgemm_op plain_gemm(const det_flinear& lin, int dtype, size_t t) {
    det_fgemm_op g{};
    g.lin = &lin;
    g.dtype = dtype;
    g.nseg = 1;
    g.seg_end[0] = lin.N;
    g.glu_from = lin.N;
    g.M = (int)t;
    return g;
}
}  // namespace

// ---------------------------------------------------------------------------------------------------- configuration
// Mixer and feed-forward of a serial layer.
static void read_serial(const std::string& type, const Json& x, const Json& e, LayerSpec& l) {
    MixerSpec& m = l.mixer;
    if (type == "attention") {
        m.kind = MixerKind::Attention;
        m.heads = x.size("heads");
        m.kv_heads = x.size("kv_heads");
        m.dim = x.size("dim");
        m.vdim = x.size("vdim");
        m.scale = (float)x.number("scale");
        const Json& rot = x.at("rot");
        m.rot_base = rot.number("base");
        m.rot_dims = rot.size("dims");
        if (m.heads == 0 || m.kv_heads == 0 || m.dim == 0 || m.vdim == 0) bad("head counts and sizes must be positive");
        if (m.heads % m.kv_heads) bad("'heads' must be a multiple of 'kv_heads'");
        if (m.dim > 1024 || m.vdim > 1024) bad("head sizes up to 1024 are supported");
        if (m.rot_dims % 2 || m.rot_dims > m.dim) bad("'rot.dims' must be even and at most dim");
        if (m.vdim % 2) bad("'vdim' must be even: values are rotated");
    } else if (type == "mingru") {
        m.kind = MixerKind::MinGru;
        m.width = x.size("width");
        if (m.width == 0) bad("'width' must be positive");
    } else {
        bad("unknown mixer '" + type + "'");
    }
    if (!e.has("mlp")) return;
    const Json& f = e.at("mlp");
    const std::string& kind = f.string("kind");
    if (kind == "dense") {
        l.ff = f.size("ff");
        if (l.ff == 0) bad("'ff' must be positive");
    } else if (kind == "moe") {
        const Json& r = f.at("router");
        l.moe.experts = r.size("experts");
        l.moe.identity = r.has("identity") ? r.size("identity") : 0;
        l.moe.top = r.size("top");
        l.moe.ff = f.at("expert").size("ff");
        if (f.has("shared")) {
            l.moe.shared = f.at("shared").size("ff");
            if (l.moe.shared == 0) bad("'shared.ff' must be positive");
        }
        if (l.moe.experts == 0 || l.moe.ff == 0) bad("a mixture needs experts");
        if (l.moe.outputs() > DET_MAX_ROUTER) bad("a router has at most " + std::to_string(DET_MAX_ROUTER) + " outputs");
        if (l.moe.top == 0 || l.moe.top > l.moe.outputs()) bad("'router.top' must be between 1 and the number of outputs");
    } else {
        bad("unknown feed-forward '" + kind + "'");
    }
}

HybridConfig HybridConfig::from_json(const Json& j) {
    HybridConfig c;
    c.vocab = j.size("vocab");
    c.width = j.size("width");
    c.eps = (float)j.at("norm").number("eps");
    c.softcap = j.has("logit_softcap") ? (float)j.number("logit_softcap") : 0.0f;
    if (c.vocab == 0 || c.width == 0) bad("vocab and width must be positive");
    c.serial = j.has("architecture") && j.string("architecture") == "Dopipel";
    if (c.serial && j.has("canon")) {
        c.taps = j.at("canon").size("taps");
        if (c.taps == 0 || c.taps > DET_MAX_TAPS) bad("'canon.taps' must be between 1 and " + std::to_string(DET_MAX_TAPS));
    }
    const Json& layers = j.at("layers");
    if (layers.kind != Json::Array || layers.items.empty()) bad("'layers' is not a list of layers");
    for (size_t i = 0; i < layers.items.size(); i++) {
        const Json& e = layers.items[i];
        LayerSpec l;
        l.weights = i;
        MixerSpec& m = l.mixer;
        try {
            const std::string& type = e.string("type");
            const Json& x = e.at("mixer");
            if (c.serial) {
                read_serial(type, x, e, l);
                c.layers.push_back(l);
                continue;
            }
            m.heads = x.size("heads");
            m.dim = x.size("dim");
            if (type == "gla") {
                m.kind = MixerKind::Gla;
                m.vdim = x.size("vdim");
                m.tau = (float)x.number("tau");
                if (!(m.tau > 0.0f)) bad("'tau' must be positive");
            } else if (type == "wkv") {
                m.kind = MixerKind::Wkv;
                m.vdim = m.dim;
            } else if (type == "latent_attention") {
                m.kind = MixerKind::Latent;
                m.vdim = x.size("vdim");
                m.q_rank = x.size("q_rank");
                m.kv_rank = x.size("kv_rank");
                m.rot_dim = x.size("rot_dim");
                m.scale = (float)x.number("scale");
                const Json& rot = x.at("rot");
                m.rot_base = rot.number("base");
                m.rot_dims = rot.size("dims");
                if (m.rot_dims % 2 || m.rot_dims > m.rot_dim) bad("'rot.dims' must be even and at most rot_dim");
                if (x.has("mask")) {
                    m.window = x.at("mask").size("size");
                    if (m.window == 0) bad("'mask.size' must be positive");
                }
            } else {
                bad("unknown mixer '" + type + "'");
            }
            if (m.heads == 0 || m.dim == 0 || m.vdim == 0) bad("head counts and sizes must be positive");
            if (e.has("mlp")) {
                const std::string& kind = e.at("mlp").string("kind");
                if (kind != "dense") bad("unknown feed-forward '" + kind + "'");
                l.ff = e.at("mlp").size("ff");
                if (l.ff == 0) bad("'ff' must be positive");
            }
            if (e.has("weights_of")) {
                l.weights = e.size("weights_of");
                if (l.weights >= layers.items.size()) bad("'weights_of' names no layer");
            }
        } catch (const std::exception& ex) {
            bad("layer " + std::to_string(i) + ": " + ex.what());
        }
        c.layers.push_back(l);
    }
    size_t from = 0, to = 0, times = 1;
    if (c.serial && j.has("loop")) {
        const Json& loop = j.at("loop");
        from = loop.size("start");
        to = loop.size("stop");
        times = c.passes = loop.size("times");
        if (from >= to || to > c.layers.size() || times == 0) bad("'loop' names no layers or no pass");
    }
    for (size_t i = 0; i < from; i++) c.runs.push_back({i, -1});
    for (size_t p = 0; p < times; p++)
        for (size_t i = from; i < to; i++) c.runs.push_back({i, i == from ? (int)p : -1});
    for (size_t i = to; i < c.layers.size(); i++) c.runs.push_back({i, -1});
    for (size_t i = 0; i < c.layers.size(); i++) {
        size_t o = c.layers[i].weights;
        for (size_t hops = 0; c.layers[o].weights != o; o = c.layers[o].weights)
            if (++hops > c.layers.size()) bad("layer " + std::to_string(i) + ": 'weights_of' goes in a circle");
        const LayerSpec& own = c.layers[o];
        const MixerSpec &n = own.mixer, &m = c.layers[i].mixer;
        if (n.kind != m.kind || n.heads != m.heads || n.dim != m.dim || n.vdim != m.vdim || n.q_rank != m.q_rank ||
            n.kv_rank != m.kv_rank || n.rot_dim != m.rot_dim || own.ff != c.layers[i].ff)
            bad("layer " + std::to_string(i) + ": 'weights_of' names a layer of other sizes");
        c.layers[i].weights = o;
    }
    return c;
}

// ---------------------------------------------------------------------------------------------------- tensor sources
namespace {
struct FileSource : TensorSource {
    std::shared_ptr<SafeTensors> f;
    const SafeTensor& get(const std::string& name) {
        const SafeTensor* t = f->find(name);
        if (!t) bad("missing tensor " + name);
        return *t;
    }
    void matrix(const std::string& name, size_t rows, size_t cols, uint16_t* out) override {
        const SafeTensor& t = get(name);
        if (t.shape != std::vector<size_t>{rows, cols})
            bad(name + ": expected a " + std::to_string(rows) + " x " + std::to_string(cols) + " matrix");
        if (t.dtype != "BF16") bad(name + ": expected bfloat16, found " + t.dtype);
        std::memcpy(out, t.data, t.bytes);
        for (size_t i = 0; i < rows * cols; i++)
            if ((out[i] & 0x7F80) == 0x7F80) bad(name + ": not finite");
    }
    std::vector<float> vector(const std::string& name, size_t n) override {
        const SafeTensor& t = get(name);
        if (t.n_elems() != n) bad(name + ": expected " + std::to_string(n) + " values");
        std::vector<float> v(n);
        if (t.dtype == "F32") std::memcpy(v.data(), t.data, t.bytes);
        else if (t.dtype == "BF16")
            for (size_t i = 0; i < n; i++) {
                uint16_t b;
                std::memcpy(&b, t.data + 2 * i, 2);
                v[i] = bf16_to_f32(b);
            }
        else bad(name + ": expected bfloat16 or float32, found " + t.dtype);
        for (float x : v)
            if (!std::isfinite(x)) bad(name + ": not finite");
        return v;
    }
    size_t rows_of(const std::string& name, size_t cols) override {
        const SafeTensor& t = get(name);
        if (t.shape.size() != 2 || t.shape[1] != cols) bad(name + ": expected a matrix of width " + std::to_string(cols));
        return t.shape[0];
    }
};
struct SynthSource : TensorSource {
    Backend* bk;
    uint64_t seed, next = 1;
    size_t rank = 64;      // of the low-rank decay projections
    void matrix(const std::string&, size_t rows, size_t cols, uint16_t* out) override {
        const uint64_t tid = next++;
        for (size_t i = 0; i < rows * cols; i++) out[i] = f32_to_bf16(draw_normal(seed, tid, i, WEIGHT_STD));
    }
    std::vector<float> vector(const std::string& name, size_t n) override {
        // unit norms, a router's choice left to its scores; the other small vectors (mixes, biases, bonuses, sinks) are drawn
        const bool norm = name.find("norm") != std::string::npos, choice = name.find("correction") != std::string::npos;
        const uint64_t tid = next++;
        std::vector<float> v(n, choice ? 0.0f : 1.0f);
        if (!norm && !choice)
            for (size_t i = 0; i < n; i++) v[i] = draw_unit(seed, tid, i);
        return v;
    }
    size_t rows_of(const std::string&, size_t) override { return rank; }
    bool on_device(const std::string&, size_t rows, size_t cols, uint16_t* out) override {
        if (!out) return false;
        bk->synth_bf16(seed, next++, rows * cols, out);
        return true;
    }
};

// Rows of a packed linear: tensor rows go to given physical rows (stride `step`) at a column offset.
class Packer {
  public:
    Packer(Backend* bk, TensorSource& src, size_t n, size_t k) : bk_(bk), src_(src) {
        lin_.n = n;
        lin_.k = k;
        lin_.ld = round8(k);
        lin_.w = bk->alloc<uint16_t>(n * lin_.ld);   // zero-filled
    }
    void part(const std::string& name, size_t rows, size_t cols, size_t row0, size_t step = 1, size_t col0 = 0) {
        if (step == 1 && cols == lin_.ld && src_.on_device(name, rows, cols, lin_.w.ptr_at(row0 * lin_.ld))) return;
        tmp_.resize(rows * cols);
        src_.matrix(name, rows, cols, tmp_.data());
        if (host_.empty()) host_.assign(lin_.n * lin_.ld, 0);
        for (size_t r = 0; r < rows; r++)
            std::memcpy(&host_[(row0 + r * step) * lin_.ld + col0], &tmp_[r * cols], cols * 2);
        filled_.push_back({row0, step, rows});
    }
    // a stack of `groups` linears of equal size, the next call's rows of each being the tensors name(i)
    template <class Name>
    FLinear stack(size_t groups, size_t rows, size_t cols, Name name) {
        lin_.groups = groups;
        if (!src_.on_device(name(0), lin_.n, cols, cols == lin_.ld ? lin_.w.ptr() : nullptr))
            for (size_t i = 0; i < groups; i++) part(name(i), rows, cols, i * rows);
        return finish();
    }
    FLinear finish(std::vector<int> seg_end = {}) {
        if (!host_.empty()) {
            size_t lo = lin_.n, hi = 0;   // rows written on the host form one span (device-filled parts lie outside it)
            for (const auto& f : filled_) {
                lo = std::min(lo, f[0]);
                hi = std::max(hi, f[0] + (f[2] - 1) * f[1] + 1);
            }
            bk_->write(lin_.w, lo * lin_.ld, host_.data() + lo * lin_.ld, (hi - lo) * lin_.ld);
            bk_->sync();   // the staging buffer dies here
        }
        lin_.seg_end = std::move(seg_end);
        if (lin_.seg_end.empty()) lin_.seg_end = {(int)lin_.n};
        bk_->f_linear_ready(lin_);
        return std::move(lin_);
    }

  private:
    Backend* bk_;
    TensorSource& src_;
    FLinear lin_;
    std::vector<uint16_t> host_, tmp_;
    std::vector<std::array<size_t, 3>> filled_;
};
}  // namespace

// ---------------------------------------------------------------------------------------------------- loading
static std::shared_ptr<HybridWeights> load_layer(const HybridConfig& c, size_t i, TensorSource& src, Backend* bk, bool synthetic) {
    auto wp = std::make_shared<HybridWeights>();
    HybridWeights& w = *wp;
    const LayerSpec& l = c.layers[i];
    const MixerSpec& m = l.mixer;
    const std::string p = "l" + std::to_string(i) + ".", mix = p + "mix.", mlp = p + "mlp.";
    const size_t W = c.width, qk = m.heads * m.dim, vo = m.width_out();
    auto vec = [&](const std::string& name, size_t n) { return bk->upload(src.vector(name, n)); };
    w.norm1 = vec(p + "norm1", W);

    struct Part {
        std::string name;
        size_t rows;
    };
    std::vector<Part> parts;
    switch (m.kind) {
        case MixerKind::Gla:
            w.rank = src.rows_of(mix + "a1", W);
            parts = {{"q", qk}, {"k", qk}, {"v", vo}, {"g", vo}, {"a1", w.rank}};
            break;
        case MixerKind::Wkv:
            w.rank = src.rows_of(mix + "w1", W);
            parts = {{"r", qk}, {"k", qk}, {"v", vo}, {"g", vo}, {"w1", w.rank}};
            break;
        case MixerKind::Latent:
            parts = {{"dq", m.q_rank}, {"dkv", m.kv_rank + m.rot_dim}, {"g", vo}};
            break;
        default: throw std::logic_error("not a mixer of a parallel layer");
    }
    for (size_t q = 0; q < parts.size(); q++) {
        w.off[q] = w.plain;
        w.plain += parts[q].rows;
    }
    Packer in(bk, src, w.plain + 2 * l.ff, W);
    for (size_t q = 0; q < parts.size(); q++) in.part(mix + parts[q].name, parts[q].rows, W, w.off[q]);
    if (l.ff) {
        if (synthetic && W % 8 == 0) {
            in.part(mlp + "gate", 2 * l.ff, W, w.plain);   // a random matrix needs no interleaving
        } else {
            in.part(mlp + "gate", l.ff, W, w.plain, 2);
            in.part(mlp + "up", l.ff, W, w.plain + 1, 2);
        }
    }
    std::vector<int> ends;      // wkv: every part reads an input of its own
    if (m.kind == MixerKind::Wkv)
        for (size_t q = 1; q < parts.size(); q++) ends.push_back((int)w.off[q]);
    ends.push_back((int)w.plain);
    if (l.ff) ends.push_back((int)(w.plain + 2 * l.ff));
    w.in = in.finish(ends);

    w.out_ff = round8(vo);
    Packer out(bk, src, W, l.ff ? w.out_ff + l.ff : vo);
    if (synthetic && vo % 8 == 0 && l.ff % 8 == 0) {
        out.part(mix + "o", W, vo + l.ff, 0);
    } else {
        out.part(mix + "o", W, vo, 0);
        if (l.ff) out.part(mlp + "down", W, l.ff, 0, 1, w.out_ff);
    }
    w.out = out.finish();

    if (m.kind == MixerKind::Latent) {
        w.dq_norm = vec(mix + "dq.norm", m.q_rank);
        w.dkv_norm = vec(mix + "dkv.norm", m.kv_rank);
        w.sink = vec(mix + "sink", m.heads);
        Packer uq(bk, src, m.heads * (m.dim + m.rot_dim), m.q_rank);
        uq.part(mix + "uq", m.heads * (m.dim + m.rot_dim), m.q_rank, 0);
        w.uq = uq.finish();
        Packer ukv(bk, src, qk + vo, m.kv_rank);
        ukv.part(mix + "uk", qk, m.kv_rank, 0);
        ukv.part(mix + "uv", vo, m.kv_rank, qk);
        w.ukv = ukv.finish();
        return wp;
    }
    const bool gla = m.kind == MixerKind::Gla;
    Packer decay(bk, src, qk, w.rank);
    decay.part(mix + (gla ? "a2" : "w2"), qk, w.rank, 0);
    w.decay = decay.finish();
    w.decay_bias = vec(mix + (gla ? "a2.b" : "w0"), qk);
    if (gla) {
        // one norm weight for all heads: repeated, so that the kernels index by channel in either mixer
        const std::vector<float> n = src.vector(mix + "norm", m.vdim);
        std::vector<float> all;
        for (size_t h = 0; h < m.heads; h++) all.insert(all.end(), n.begin(), n.end());
        w.head_norm = bk->upload(all);
        bk->sync();
    } else {
        w.head_norm = vec(mix + "norm", vo);
        w.bonus = vec(mix + "u", qk);
        std::vector<float> mu;
        for (const char* n : {"r", "k", "v", "g", "w"}) {
            const std::vector<float> v = src.vector(mix + "mu." + n, W);
            mu.insert(mu.end(), v.begin(), v.end());
        }
        w.mu = bk->upload(mu);
        bk->sync();
    }
    return wp;
}

// The tensors of a serial layer.
static std::shared_ptr<HybridWeights> load_serial(const HybridConfig& c, size_t i, TensorSource& src, Backend* bk, bool synthetic) {
    auto wp = std::make_shared<HybridWeights>();
    HybridWeights& w = *wp;
    const LayerSpec& l = c.layers[i];
    const MixerSpec& m = l.mixer;
    const std::string p = "l" + std::to_string(i) + ".", mix = p + "mix.", mlp = p + "mlp.";
    const size_t W = c.width, vo = m.width_out();
    auto vec = [&](const std::string& name, size_t n) { return bk->upload(src.vector(name, n)); };
    w.norm1 = vec(p + "norm1", W);
    w.norm1b = vec(p + "norm1b", W);
    w.scale1 = vec(p + "ls1", W);
    if (c.taps) {
        const std::vector<float> v = src.vector(p + "canon1", W * c.taps);      // [width][taps]
        std::vector<float> t(v.size());
        for (size_t ch = 0; ch < W; ch++)
            for (size_t k = 0; k < c.taps; k++) t[k * W + ch] = v[ch * c.taps + k];
        w.conv = bk->upload(t);
        bk->sync();
    }
    struct Part {
        std::string name;
        size_t rows;
        bool bias;
    };
    std::vector<Part> parts;
    if (m.kind == MixerKind::Attention)
        parts = {{"q", m.heads * m.dim, true}, {"k", m.kv_heads * m.dim, true}, {"v", m.kv_heads * m.vdim, true}, {"g", m.heads, false}};
    else
        parts = {{"z", m.width, true}, {"x", m.width, true}, {"g", m.width, false}};
    std::vector<float> bias;
    for (size_t q = 0; q < parts.size(); q++) {
        w.off[q] = w.plain;
        w.plain += parts[q].rows;
        std::vector<float> b(parts[q].rows, 0.0f);
        if (parts[q].bias) b = src.vector(mix + parts[q].name + ".b", parts[q].rows);
        bias.insert(bias.end(), b.begin(), b.end());
    }
    w.in_bias = bk->upload(bias);
    bk->sync();
    Packer in(bk, src, w.plain, W);
    for (size_t q = 0; q < parts.size(); q++) in.part(mix + parts[q].name, parts[q].rows, W, w.off[q]);
    w.in = in.finish();
    Packer out(bk, src, W, vo);
    out.part(mix + "o", W, vo, 0);
    w.out = out.finish();
    if (m.kind == MixerKind::Attention) w.out_bias = vec(mix + "o.b", W);
    bk->sync();
    if (!l.ff && !l.moe.experts) return wp;

    w.norm2 = vec(p + "norm2", W);
    w.norm2b = vec(p + "norm2b", W);
    w.scale2 = vec(p + "ls2", W);
    if (l.ff) {
        Packer fi(bk, src, 2 * l.ff, W);
        if (synthetic && W % 8 == 0) {
            fi.part(mlp + "gate", 2 * l.ff, W, 0);       // a random matrix needs no interleaving
        } else {
            fi.part(mlp + "gate", l.ff, W, 0, 2);
            fi.part(mlp + "up", l.ff, W, 1, 2);
        }
        w.ff_in = fi.finish();
        Packer fo(bk, src, W, l.ff);
        fo.part(mlp + "down", W, l.ff, 0);
        w.ff_out = fo.finish();
        bk->sync();
        return wp;
    }
    const MoeSpec& e = l.moe;
    w.ff_plain = e.outputs() + (e.shared ? 1 : 0);
    Packer fi(bk, src, w.ff_plain + e.shared, W);
    fi.part(mlp + "router", e.outputs(), W, 0);
    if (e.shared) {
        fi.part(mlp + "shared.sg", 1, W, e.outputs());
        fi.part(mlp + "shared.up", e.shared, W, w.ff_plain);
        w.ff_in = fi.finish({(int)w.ff_plain, (int)(w.ff_plain + e.shared)});
        Packer fo(bk, src, W, e.shared);
        fo.part(mlp + "shared.down", W, e.shared, 0);
        w.ff_out = fo.finish();
    } else {
        w.ff_in = fi.finish();
    }
    w.correction = vec(mlp + "correction", e.outputs());
    w.up = Packer(bk, src, e.experts * e.ff, W).stack(e.experts, e.ff, W, [&](size_t k) { return mlp + "e" + std::to_string(k) + ".up"; });
    w.down = Packer(bk, src, e.experts * W, e.ff).stack(e.experts, W, e.ff, [&](size_t k) { return mlp + "e" + std::to_string(k) + ".down"; });
    bk->sync();
    return wp;
}

static HybridCache make_cache(const HybridConfig& c, Backend* bk, Dtype dtype, size_t ctx, size_t max_batch) {
    HybridCache s;
    for (const LayerRun& run : c.runs) {
        const MixerSpec& m = c.layers[run.layer].mixer;
        FloatState f;
        if (c.serial) {
            if (c.taps > 1) f.prev = bk->alloc<float>((c.taps - 1) * c.width);
            if (m.kind == MixerKind::MinGru) {
                f.s = bk->alloc<float>(m.width);
            } else {
                f.cap = ctx;
                f.cache = bk->alloc<uint8_t>(ctx * (size_t)det_f_attn_ld((int)m.kv_heads, (int)m.dim, (int)m.vdim) * dtype_bytes(dtype));
            }
        } else if (m.kind == MixerKind::Latent) {
            // a step of max_batch tokens still needs the window before its first one
            f.cap = m.window ? std::min(ctx, m.window - 1 + max_batch) : ctx;
            f.cache = bk->alloc<uint8_t>(f.cap * (size_t)det_f_latent_ld((int)m.kv_rank, (int)m.rot_dim) * dtype_bytes(dtype));
        } else {
            f.s = bk->alloc<float>(m.heads * m.dim * m.vdim);
            if (m.kind == MixerKind::Wkv) f.prev = bk->alloc<float>(c.width);
        }
        s.layers.push_back(std::move(f));
    }
    return s;
}

// Rotation table [position][dims / 2], angle position * base^(-2i / dims): binary64, rounded once.
void HybridModel::add_rope(double base, size_t dims) {
    for (const Rope& r : ropes_)
        if (r.base == base && r.dims == dims) return;
    const size_t half = dims / 2;
    std::vector<float> rc(max_ctx * half + 1), rs(max_ctx * half + 1);
    for (size_t i = 0; i < half; i++) {
        const double f = std::pow(base, -2.0 * (double)i / (double)dims);
        for (size_t p = 0; p < max_ctx; p++) {
            rc[p * half + i] = (float)std::cos((double)p * f);
            rs[p * half + i] = (float)std::sin((double)p * f);
        }
    }
    ropes_.push_back(Rope{base, dims, backend->upload(rc), backend->upload(rs)});
    backend->sync();
}

std::unique_ptr<HybridModel> HybridModel::load(const HybridConfig& cfg, TensorSource& src, Backend* bk, size_t max_ctx,
                                               size_t max_batch, Dtype dtype) {
    if (max_ctx == 0 || max_batch == 0) bad("the context and the batch must be positive");
    auto mp = std::make_unique<HybridModel>();
    HybridModel& m = *mp;
    m.cfg = cfg;
    m.backend = bk;
    m.dtype = dtype;
    m.max_ctx = max_ctx;
    m.max_batch = max_batch;
    const bool synthetic = dynamic_cast<SynthSource*>(&src) != nullptr;
    const size_t W = cfg.width;
    m.embed_ = bk->alloc<uint16_t>(cfg.vocab * W);
    if (!src.on_device("embed", cfg.vocab, W, m.embed_.ptr())) {
        std::vector<uint16_t> e(cfg.vocab * W);
        src.matrix("embed", cfg.vocab, W, e.data());
        bk->write(m.embed_, 0, e.data(), e.size());
        bk->sync();
    }
    m.weights_.resize(cfg.layers.size());
    for (size_t i = 0; i < cfg.layers.size(); i++)
        if (cfg.layers[i].weights == i) m.weights_[i] = (cfg.serial ? load_serial : load_layer)(cfg, i, src, bk, synthetic);
    for (size_t i = 0; i < cfg.layers.size(); i++) m.weights_[i] = m.weights_[cfg.layers[i].weights];
    m.final_norm_ = bk->upload(src.vector("final.norm", W));
    bk->sync();
    Packer head(bk, src, cfg.vocab, W);
    head.part("head", cfg.vocab, W, 0);
    m.head_lin_ = head.finish();

    for (const LayerSpec& l : cfg.layers) {
        const MixerSpec& x = l.mixer;
        if (x.kind == MixerKind::Latent || x.kind == MixerKind::Attention) m.add_rope(x.rot_base, x.rot_dims);
        if (x.kind == MixerKind::Attention) m.add_rope(x.rot_base, x.vdim);      // values turn over all of their dimensions
    }
    m.bound_ = make_cache(cfg, bk, dtype, max_ctx, max_batch);

    size_t groups = 1, ldy = 1, cat = 8, q = 1;
    m.ld_cq_ = 8;
    for (size_t i = 0; i < cfg.layers.size(); i++) {
        const HybridWeights& w = *m.weights_[i];
        const MixerSpec& x = cfg.layers[i].mixer;
        ldy = std::max(ldy, round8(w.plain));
        ldy = std::max(ldy, round8(w.ff_plain));
        cat = std::max({cat, w.out.ld, w.ff_out.ld});
        if (x.kind == MixerKind::Wkv) groups = 6;
        if (x.kind == MixerKind::Latent) {
            m.ld_cq_ = std::max(m.ld_cq_, round8(x.q_rank));
            q = std::max(q, x.heads * (x.dim + x.rot_dim));
        }
        if (x.kind == MixerKind::Attention) q = std::max(q, (size_t)det_f_attn_q_ld((int)x.heads, (int)x.dim));
    }
    m.ld_in_ = round8(W);
    const size_t e = dtype_bytes(dtype);
    m.in_ = bk->alloc<uint8_t>(groups * max_batch * m.ld_in_ * e);
    m.cat_ = bk->alloc<uint8_t>(max_batch * cat * e);
    m.cq_ = bk->alloc<uint8_t>(max_batch * m.ld_cq_ * e);
    m.y_ = bk->alloc<float>(max_batch * ldy);
    m.q_ = bk->alloc<float>(max_batch * q);
    m.ids_ = bk->alloc<int32_t>(max_batch);
    m.rows_ = bk->alloc<int32_t>(max_batch);
    if (cfg.serial) {
        m.res_ = bk->alloc<float>(max_batch * W);
        m.rstd_ = bk->alloc<float>(max_batch);
    }
    if (cfg.passes) {
        Packer mix(bk, src, W, 2 * W);
        mix.part("loop.in", W, 2 * W, 0);
        m.loop_lin_ = mix.finish();
        m.loop_step_ = bk->upload(src.vector("loop.step", cfg.passes * W));
        bk->sync();
        m.ld_pair_ = round8(2 * W);
        m.pair_ = bk->alloc<uint8_t>(max_batch * m.ld_pair_ * e);
    }
    m.x = bk->alloc<float>(max_batch * W);
    m.logits_buf = bk->alloc<float>(cfg.vocab);
    return mp;
}

std::unique_ptr<HybridModel> HybridModel::load_dir(const std::string& dir, const Json& config, Backend* bk, size_t max_ctx,
                                                   size_t max_batch, Dtype dtype) {
    FileSource src;
    src.f = SafeTensors::open(dir + "/model.safetensors");
    return load(HybridConfig::from_json(config), src, bk, max_ctx, max_batch, dtype);
}
std::unique_ptr<HybridModel> HybridModel::load_synthetic(const Json& config, uint64_t seed, Backend* bk, size_t max_ctx,
                                                         size_t max_batch, Dtype dtype) {
    SynthSource src;
    src.bk = bk;
    src.seed = seed;
    return load(HybridConfig::from_json(config), src, bk, max_ctx, max_batch, dtype);
}

size_t HybridModel::weight_bytes() const {
    auto bytes = [](const FLinear& l) { return l.n * l.ld * 2; };
    size_t s = bytes(head_lin_) + cfg.passes * bytes(loop_lin_);
    for (const LayerRun& run : cfg.runs) {
        const HybridWeights& w = *weights_[run.layer];
        const MoeSpec& m = cfg.layers[run.layer].moe;
        s += bytes(w.in) + bytes(w.out) + bytes(w.decay) + bytes(w.uq) + bytes(w.ukv) + bytes(w.ff_in) + bytes(w.ff_out);
        if (m.experts) s += (bytes(w.up) + bytes(w.down)) / m.experts * std::min(m.top, m.experts);
    }
    return s;
}

// ---------------------------------------------------------------------------------------------------- sequences
std::unique_ptr<SeqCache> HybridModel::new_sequence(size_t ctx) {
    if (ctx > max_ctx) bad("a sequence's context exceeds the model's");   // the rotation tables end there
    return std::make_unique<HybridCache>(make_cache(cfg, backend, dtype, ctx, max_batch));
}
void HybridModel::swap_sequence(SeqCache& s) { std::swap(bound_.layers, dynamic_cast<HybridCache&>(s).layers); }
// Cache rows need no clearing: a position only reads rows its own sequence wrote.
void HybridModel::clear_sequence(SeqCache& s) {
    for (FloatState& f : dynamic_cast<HybridCache&>(s).layers) {
        if (f.s.ptr()) backend->zero(f.s);
        if (f.prev.ptr()) backend->zero(f.prev);
    }
}
std::vector<std::unique_ptr<RowSet>> HybridModel::make_rowsets(const std::vector<SeqCache*>& seqs) {
    std::vector<std::unique_ptr<RowSet>> sets;
    for (size_t i = 0; i < cfg.runs.size(); i++) {
        std::vector<const FloatState*> fs;
        for (SeqCache* s : seqs) {
            fs.push_back(&dynamic_cast<HybridCache&>(*s).layers[i]);
            if (fs.back()->cap != fs[0]->cap) bad("the sequences of a batch must have caches of one size");
        }
        sets.push_back(backend->make_slots(std::move(fs)));
    }
    return sets;
}

// ---------------------------------------------------------------------------------------------------- network
std::string HybridModel::embed_rows(const int32_t* ids, size_t t) {
    for (size_t i = 0; i < t; i++)
        if (ids[i] < 0 || (size_t)ids[i] >= cfg.vocab)
            return "token id " + std::to_string(ids[i]) + " is outside the embedding table (" + std::to_string(cfg.vocab) + " rows)";
    backend->write(ids_, 0, ids, t);
    backend->embed(embed_.ptr(), 30, ids_, t, cfg.width, x);
    return "";
}

const HybridModel::Rope& HybridModel::rope(double base, size_t dims) const {
    for (const Rope& r : ropes_)
        if (r.base == base && r.dims == dims) return r;
    throw std::logic_error("no rotation table");
}

// norm1 and every projection of the normalised row: mixer parts into y_, SwiGLU product behind the mixer's columns of cat_
void HybridModel::run_in(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq) {
    const det_flinear lin = w.in.view();
    det_fgemm_op g{};
    g.lin = &lin;
    g.dtype = (int)dtype;
    g.x = in_.ptr();
    g.ldx = (int)ld_in_;
    g.group_stride = (long long)(max_batch * ld_in_);
    g.M = (int)t;
    g.glu_from = (int)w.plain;
    g.nseg = (int)w.in.seg_end.size();
    for (int i = 0; i < g.nseg; i++) {
        g.seg_end[i] = w.in.seg_end[i];
        g.seg_in[i] = l.mixer.kind == MixerKind::Wkv ? i : 0;     // r, k, v, g, w1, then the feed-forward on h itself
    }
    if (l.mixer.kind == MixerKind::Wkv) {
        det_fnorm_op n{};
        n.x = x.ptr();
        n.w = w.norm1.ptr();
        n.eps = cfg.eps;
        n.M = (int)t;
        n.n = (int)cfg.width;
        n.dtype = (int)dtype;
        n.out = in_.ptr();
        n.ld = (int)ld_in_;
        n.group_stride = g.group_stride;
        n.nmix = 5;
        n.mu = w.mu.ptr();
        n.seq = seq;
        backend->f_norm(n);
    } else {
        g.norm_x = x.ptr();
        g.norm_w = w.norm1.ptr();
        g.eps = cfg.eps;
    }
    g.y = y_.ptr();
    g.ldy = (int)round8(w.plain);
    g.h = cat_.ptr() + w.out_ff * dtype_bytes(dtype);
    g.ldh = (int)w.out.ld;
    backend->f_gemm(g);
}

void HybridModel::mixer_recurrent(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq) {
    const MixerSpec& m = l.mixer;
    const det_flinear w2 = w.decay.view();
    const bool gla = m.kind == MixerKind::Gla;
    det_frecur_op r{};
    r.heads = (int)m.heads;
    r.dk = (int)m.dim;
    r.dv = (int)m.vdim;
    r.rank = (int)w.rank;
    r.M = (int)t;
    r.dtype = (int)dtype;
    r.y = y_.ptr();
    r.ldy = (int)round8(w.plain);
    r.q_off = (int)w.off[0];
    r.k_off = (int)w.off[1];
    r.v_off = (int)w.off[2];
    r.gate_off = (int)w.off[3];
    r.low_off = (int)w.off[4];
    r.q_scale = gla ? (float)(1.0 / std::sqrt((double)m.dim)) : 1.0f;
    r.decay = gla ? DET_DECAY_SIGMOID : DET_DECAY_EXP;
    r.tau = m.tau;
    r.w2 = &w2;
    r.bias = w.decay_bias.ptr();
    r.u = gla ? nullptr : w.bonus.ptr();
    r.norm = w.head_norm.ptr();
    r.eps = cfg.eps;
    r.out = cat_.ptr();
    r.ldo = (int)w.out.ld;
    r.seq = seq;
    backend->f_recur(r);
}

void HybridModel::mixer_latent(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq, size_t cap, size_t max_pos) {
    const MixerSpec& m = l.mixer;
    const det_flinear uq = w.uq.view(), ukv = w.ukv.view();
    const Rope& rp = rope(m.rot_base, m.rot_dims);
    det_flatent_op a{};
    a.heads = (int)m.heads;
    a.dim = (int)m.dim;
    a.rot_dim = (int)m.rot_dim;
    a.rot_dims = (int)m.rot_dims;
    a.vdim = (int)m.vdim;
    a.q_rank = (int)m.q_rank;
    a.kv_rank = (int)m.kv_rank;
    a.window = (int)m.window;
    a.scale = m.scale;
    a.cap = (int)cap;
    a.M = (int)t;
    a.dtype = (int)dtype;
    a.y = y_.ptr();
    a.ldy = (int)round8(w.plain);
    a.dq_off = (int)w.off[0];
    a.dkv_off = (int)w.off[1];
    a.gate_off = (int)w.off[2];
    a.dq_norm = w.dq_norm.ptr();
    a.dkv_norm = w.dkv_norm.ptr();
    a.eps = cfg.eps;
    a.rope_cos = rp.cos.ptr();
    a.rope_sin = rp.sin.ptr();
    a.cq = cq_.ptr();
    a.ldcq = (int)ld_cq_;
    a.q = q_.ptr();
    a.ldq = (int)w.uq.n;
    a.wkv = &ukv;
    a.sink = w.sink.ptr();
    a.out = cat_.ptr();
    a.ldo = (int)w.out.ld;
    a.max_pos = (int)max_pos;
    a.seq = seq;
    backend->f_latent_prep(a);
    det_fgemm_op g{};
    g.lin = &uq;
    g.dtype = (int)dtype;
    g.x = cq_.ptr();
    g.ldx = (int)ld_cq_;
    g.nseg = 1;
    g.seg_end[0] = (int)w.uq.n;
    g.glu_from = (int)w.uq.n;
    g.M = (int)t;
    g.y = q_.ptr();
    g.ldy = (int)w.uq.n;
    backend->f_gemm(g);
    backend->f_latent_attn(a, max_ctx);
}

void HybridModel::mixer_attention(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq, size_t cap,
                                  size_t max_pos) {
    const MixerSpec& m = l.mixer;
    const Rope &rp = rope(m.rot_base, m.rot_dims), &vp = rope(m.rot_base, m.vdim);
    det_fattn_op a{};
    a.heads = (int)m.heads;
    a.kv_heads = (int)m.kv_heads;
    a.dim = (int)m.dim;
    a.vdim = (int)m.vdim;
    a.rot_dims = (int)m.rot_dims;
    a.scale = m.scale;
    a.cap = (int)cap;
    a.M = (int)t;
    a.dtype = (int)dtype;
    a.y = y_.ptr();
    a.ldy = (int)round8(w.plain);
    a.q_off = (int)w.off[0];
    a.k_off = (int)w.off[1];
    a.v_off = (int)w.off[2];
    a.gate_off = (int)w.off[3];
    a.rope_cos = rp.cos.ptr();
    a.rope_sin = rp.sin.ptr();
    a.vrope_cos = vp.cos.ptr();
    a.vrope_sin = vp.sin.ptr();
    a.q = q_.ptr();
    a.out = cat_.ptr();
    a.ldo = (int)w.out.ld;
    a.max_pos = (int)max_pos;
    a.seq = seq;
    backend->f_attn(a);
}

void HybridModel::mixer_mingru(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq) {
    det_fmingru_op r{};
    r.n = (int)l.mixer.width;
    r.M = (int)t;
    r.dtype = (int)dtype;
    r.y = y_.ptr();
    r.ldy = (int)round8(w.plain);
    r.z_off = (int)w.off[0];
    r.x_off = (int)w.off[1];
    r.gate_off = (int)w.off[2];
    r.out = cat_.ptr();
    r.ldo = (int)w.out.ld;
    r.seq = seq;
    backend->f_mingru(r);
}

// ---------------------------------------------------------------------------------------------------- layers
void HybridModel::parallel_layer(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq, size_t cap, size_t max_pos) {
    run_in(l, w, t, seq);
    if (l.mixer.kind == MixerKind::Latent) mixer_latent(l, w, t, seq, cap, max_pos);
    else mixer_recurrent(l, w, t, seq);
    const det_flinear out = w.out.view();
    det_fgemm_op g = plain_gemm(out, (int)dtype, t);
    g.x = cat_.ptr();
    g.ldx = (int)w.out.ld;
    g.y = x.ptr();
    g.ldy = (int)cfg.width;
    g.accumulate = 1;
    backend->f_gemm(g);
}

// A seam without a sublayer's result and without an output.
det_fseam_op HybridModel::seam(size_t t) const {
    det_fseam_op s{};
    s.x = x.ptr();
    s.M = (int)t;
    s.n = (int)cfg.width;
    s.eps = cfg.eps;
    s.rstd = rstd_.ptr();
    s.dtype = (int)dtype;
    return s;
}

// The residual rows in the activation type, at a column of the [residual | embedding] rows.
void HybridModel::pack_rows(size_t t, size_t col) {
    det_fseam_op s = seam(t);
    s.out = pair_.ptr() + col * dtype_bytes(dtype);
    s.ld = (int)ld_pair_;
    backend->f_seam(s);
}
// x <- W [x; x0] + step, ahead of a pass
void HybridModel::loop_entry(size_t t, int pass) {
    const det_flinear lin = loop_lin_.view();
    det_fgemm_op g = plain_gemm(lin, (int)dtype, t);
    g.x = pair_.ptr();
    g.ldx = (int)ld_pair_;
    g.y = x.ptr();
    g.ldy = (int)cfg.width;
    g.bias = loop_step_.ptr_at((size_t)pass * cfg.width);
    backend->f_gemm(g);
}

// in_ -> res_: projections with their biases, mixer, output projection
void HybridModel::serial_mixer(const LayerSpec& l, const HybridWeights& w, size_t t, const det_seq_ref& seq, size_t cap, size_t max_pos) {
    const det_flinear in = w.in.view(), out = w.out.view();
    det_fgemm_op g = plain_gemm(in, (int)dtype, t);
    g.x = in_.ptr();
    g.ldx = (int)ld_in_;
    g.y = y_.ptr();
    g.ldy = (int)round8(w.plain);
    g.bias = w.in_bias.ptr();
    backend->f_gemm(g);
    if (l.mixer.kind == MixerKind::Attention) mixer_attention(l, w, t, seq, cap, max_pos);
    else mixer_mingru(l, w, t, seq);
    g = plain_gemm(out, (int)dtype, t);
    g.x = cat_.ptr();
    g.ldx = (int)w.out.ld;
    g.y = res_.ptr();
    g.ldy = (int)cfg.width;
    g.bias = w.out_bias.ptr();
    backend->f_gemm(g);
}

// in_ -> res_
void HybridModel::serial_ff(const LayerSpec& l, const HybridWeights& w, size_t t) {
    const det_flinear in = w.ff_in.view(), out = w.ff_out.view(), up = w.up.view(), down = w.down.view();
    det_fgemm_op g = plain_gemm(in, (int)dtype, t);
    g.x = in_.ptr();
    g.ldx = (int)ld_in_;
    g.nseg = (int)w.ff_in.seg_end.size();
    for (int i = 0; i < g.nseg; i++) g.seg_end[i] = w.ff_in.seg_end[i];
    g.glu_from = (int)w.ff_plain;
    g.act = l.ff ? DET_FF_REGLU : DET_FF_RELU2;
    g.y = y_.ptr();
    g.ldy = (int)round8(w.ff_plain);
    g.h = cat_.ptr();
    g.ldh = (int)w.ff_out.ld;
    backend->f_gemm(g);
    if (l.ff) {
        g = plain_gemm(out, (int)dtype, t);
        g.x = cat_.ptr();
        g.ldx = (int)w.ff_out.ld;
        g.y = res_.ptr();
        g.ldy = (int)cfg.width;
        backend->f_gemm(g);
        return;
    }
    det_fmoe_op m{};
    m.experts = (int)l.moe.experts;
    m.identity = (int)l.moe.identity;
    m.top = (int)l.moe.top;
    m.ff = (int)l.moe.ff;
    m.n = (int)cfg.width;
    m.M = (int)t;
    m.dtype = (int)dtype;
    m.z = y_.ptr();
    m.ldz = (int)round8(w.ff_plain);
    m.correction = w.correction.ptr();
    m.x = in_.ptr();
    m.ldx = (int)ld_in_;
    m.up = &up;
    m.down = &down;
    m.shared = l.moe.shared ? &out : nullptr;
    m.hs = cat_.ptr();
    m.ldhs = (int)w.ff_out.ld;
    m.shared_gate = l.moe.shared ? (int)l.moe.outputs() : -1;
    m.out = res_.ptr();
    m.ldo = (int)cfg.width;
    backend->f_moe(m, max_batch);
}

// final norm, output rows, soft cap
void HybridModel::head(size_t t) {
    const det_flinear lin = head_lin_.view();
    det_fgemm_op g{};
    g.lin = &lin;
    g.dtype = (int)dtype;
    g.x = in_.ptr();
    g.ldx = (int)ld_in_;
    g.nseg = 1;
    g.seg_end[0] = (int)cfg.vocab;
    g.glu_from = (int)cfg.vocab;
    g.y = logits_buf.ptr();
    g.ldy = (int)cfg.vocab;
    g.softcap = cfg.softcap;
    g.norm_x = all_logits ? x.ptr() : x.ptr_at((t - 1) * cfg.width);
    g.norm_w = final_norm_.ptr();
    g.eps = cfg.eps;
    g.M = all_logits ? (int)t : 1;
    if (head_rows_) {
        if (head_rows_->empty()) return;
        backend->write(rows_, 0, head_rows_->data(), head_rows_->size());
        det_fnorm_op n{};
        n.x = x.ptr();
        n.rows = rows_.ptr();
        n.w = final_norm_.ptr();
        n.eps = cfg.eps;
        n.M = g.M = (int)head_rows_->size();
        n.n = (int)cfg.width;
        n.dtype = (int)dtype;
        n.out = in_.ptr();
        n.ld = (int)ld_in_;
        backend->f_norm(n);
        g.norm_x = nullptr;
    }
    backend->f_gemm(g);
}

void HybridModel::network(size_t pos0, size_t t, Observer* obs, const RowsCtx* rows) {
    if (obs && rows) throw std::logic_error("observers are not supported on a batched decode step");
    if (head_rows_ && head_rows_->size() > max_batch) throw std::logic_error("more logits rows than the batch holds");
    const Ctx ctx{pos0, t, backend};
    auto observe = [&](Tap::Kind kind, size_t layer, const Buf<float>& b) {
        if (!obs) return;
        Tap tap;
        tap.kind = kind;
        tap.layer = layer;
        tap.x = &b;
        obs->observe(ctx, tap);
    };
    const size_t max_pos = rows ? rows->max_pos : pos0 + t - 1;
    auto seq_of = [&](size_t ri, size_t* cap) {
        const RowSet* set = rows ? (*rows->sets)[ri].get() : nullptr;
        const FloatState& state = set ? *set->fs[0] : bound_.layers[ri];
        *cap = state.cap;
        return backend->seq_ref(state, pos0, set, rows ? rows->pos : nullptr);
    };
    // What run ri reads of the new residual rows, as the second half of the seam ahead of it.
    auto opening = [&](det_fseam_op s, size_t ri, bool in_pass) {
        if (ri == cfg.runs.size()) return s;
        if (cfg.runs[ri].pass >= 0 && !in_pass) {
            s.out = pair_.ptr();
            s.ld = (int)ld_pair_;
            return s;
        }
        const HybridWeights& w = *weights_[cfg.runs[ri].layer];
        size_t cap = 0;
        s.w = w.norm1.ptr();
        s.conv = cfg.taps ? w.conv.ptr() : nullptr;
        s.taps = (int)cfg.taps;
        s.out = in_.ptr();
        s.ld = (int)ld_in_;
        s.seq = seq_of(ri, &cap);
        return s;
    };
    if (cfg.passes) pack_rows(t, cfg.width);
    if (cfg.serial) backend->f_seam(opening(seam(t), 0, false));
    for (size_t ri = 0; ri < cfg.runs.size(); ri++) {
        observe(Tap::Residual, ri, x);
        const LayerRun& run = cfg.runs[ri];
        const LayerSpec& l = cfg.layers[run.layer];
        const HybridWeights& w = *weights_[run.layer];
        size_t cap = 0;
        const det_seq_ref seq = seq_of(ri, &cap);
        if (!cfg.serial) {
            parallel_layer(l, w, t, seq, cap, max_pos);
            continue;
        }
        if (run.pass >= 0) {
            loop_entry(t, run.pass);
            backend->f_seam(opening(seam(t), ri, true));
        }
        serial_mixer(l, w, t, seq, cap, max_pos);
        det_fseam_op s = seam(t);
        s.y = res_.ptr();
        s.ldy = (int)cfg.width;
        s.y_norm = w.norm1b.ptr();
        s.y_scale = w.scale1.ptr();
        if (l.ff || l.moe.experts) {
            s.w = w.norm2.ptr();
            s.out = in_.ptr();
            s.ld = (int)ld_in_;
            backend->f_seam(s);
            serial_ff(l, w, t);
            s = seam(t);
            s.y = res_.ptr();
            s.ldy = (int)cfg.width;
            s.y_norm = w.norm2b.ptr();
            s.y_scale = w.scale2.ptr();
        }
        backend->f_seam(opening(s, ri + 1, false));
    }
    observe(Tap::Residual, cfg.runs.size(), x);
    head(t);
    observe(Tap::Logits, 0, logits_buf);
}

}  // namespace det
