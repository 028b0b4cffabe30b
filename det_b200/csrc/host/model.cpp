// The token loop over any model.  See model.hpp for the reference map.
#include "model.hpp"
#include <algorithm>
#include <cmath>
#include <stdexcept>

namespace det {

void Model::set_all_logits(bool all) {
    backend->sync();
    const size_t n = (all ? max_batch : 1) * vocab();
    if (logits_buf.len() != n) logits_buf = backend->alloc<float>(n);
    logits_resized(n);
    all_logits = all;
}


void Model::reset() {
    backend->sync();
    pos = 0;
    clear_bound();
}

std::string Model::forward(const int32_t* ids, size_t t, Observer* obs) {
    if (t == 0 || t > max_batch)
        return "batch of " + std::to_string(t) + " tokens (1 to " + std::to_string(max_batch) + " allowed)";
    if (pos + t > max_ctx)
        return std::to_string(t) + " tokens at position " + std::to_string(pos) + " exceed the context of " +
               std::to_string(max_ctx);
    std::string e = embed_rows(ids, t);
    if (!e.empty()) return e;
    network(pos, t, obs);
    pos += t;
    return "";
}

std::string Model::forward_rows(const int32_t* ids, size_t t, const std::vector<int32_t>& want) {
    for (int32_t r : want)
        if (r < 0 || (size_t)r >= t) return "logits of row " + std::to_string(r) + " of " + std::to_string(t) + " asked for";
    const size_t n = std::max<size_t>(1, want.size()) * vocab();
    if (logits_buf.len() < n) {
        backend->sync();
        logits_buf = backend->alloc<float>(n);
        logits_resized(n);
    }
    head_rows_ = &want;
    std::string e;
    try {
        e = forward(ids, t);
    } catch (...) {
        head_rows_ = nullptr;
        throw;
    }
    head_rows_ = nullptr;
    return e;
}

std::vector<float> Model::logits() { return backend->download(logits_buf); }

std::string Model::pick(Sampling& s, int32_t& id) { return pick_row(logits_buf, s, id); }

std::string Model::pick_row(const Buf<float>& row, Sampling& s, int32_t& id) {
    if (s.greedy) {
        id = backend->argmax(row, vocab());
        return "";
    }
    if (!std::isfinite(s.inv_temp) || std::isnan(s.top_p))
        return "sampling parameters inv_temp=" + std::to_string(s.inv_temp) + " top_p=" + std::to_string(s.top_p) +
               " are not finite";
    id = backend->sample(row, vocab(), s.inv_temp, s.top_k, s.top_p, next_draw(s));
    return "";
}

uint64_t Model::next_draw(Sampling& s) {
    s.rng += 0x9E3779B97F4A7C15ull;   // splitmix64 (spec/prim.rs:207-215): the state advances once per draw
    uint64_t z = s.rng;
    z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
    z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
    return z ^ (z >> 31);
}

std::string Model::prefill(const int32_t* ids, size_t n, Observer* obs) {
    for (size_t i = 0; i < n; i += max_batch) {
        std::string e = forward(ids + i, std::min(max_batch, n - i), obs);
        if (!e.empty()) return e;
    }
    return "";
}

std::string Model::generate(const int32_t* prompt, size_t n_prompt, size_t n_new, Sampling s,
                            const std::vector<int32_t>& stop, std::vector<int32_t>& out,
                            const std::function<void(int32_t)>& on_token, Observer* obs) {
    std::string e = prefill(prompt, n_prompt, obs);
    if (!e.empty()) return e;
    out.clear();
    for (size_t i = 0; i < n_new; i++) {
        int32_t id = 0;
        e = pick(s, id);
        if (!e.empty()) return e;
        if (obs) {   // model.rs:524-538
            Tap tap;
            tap.kind = Tap::Token;
            tap.id = id;
            tap.rng = s.rng;
            obs->observe(Ctx{pos - 1, 1, backend}, tap);
        }
        out.push_back(id);
        if (on_token) on_token(id);
        if (std::find(stop.begin(), stop.end(), id) != stop.end() || i + 1 == n_new) break;
        e = forward(&id, 1, obs);
        if (!e.empty()) return e;
    }
    return "";
}

}  // namespace det
