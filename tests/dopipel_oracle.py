"""Plain implementation of the Dopipel decoder's mechanisms: test infrastructure, float64, token by token, one function per
mechanism, explicit state (so that a cut of the sequence anywhere is the same computation).  Nothing here is shared with the
product path.

  x : residual row        x0 : the token's embedding row        h : what a sublayer reads        W[out, in] applied as W @ h
"""
from __future__ import annotations

import numpy as np

from hybrid_oracle import F, rms_norm, rotate_pairs, sigmoid, silu


# ---------------------------------------------------------------------------------------------------- short convolution
def causal_conv(w, h, past):
    """w[width, taps]; past: the inputs of the earlier tokens, oldest first, zeros before the first one.  Returns what is added
    to h and the past of the next token."""
    rows = np.vstack([past, h[None]])
    return np.sum(w.T * rows, axis=0), rows[1:]


# ---------------------------------------------------------------------------------------------------- attention
def attention_weights(q, K, scale):
    s = (K @ q) * scale
    p = np.exp(s - s.max())
    return p / p.sum()


def attention_step(w, c, h, st):
    H, G, d, dv, rot = c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["rot"]
    pos = len(st["k"])
    q = (w["q"] @ h + w["q.b"]).reshape(H, d)
    k = (w["k"] @ h + w["k.b"]).reshape(G, d)
    v = (w["v"] @ h + w["v.b"]).reshape(G, dv)
    q, k = rotate_pairs(q, pos, rot["base"], rot["dims"]), rotate_pairs(k, pos, rot["base"], rot["dims"])
    st["k"].append(k)
    st["v"].append(rotate_pairs(v, pos, rot["base"], dv))
    K, V = np.array(st["k"]), np.array(st["v"])
    gate = sigmoid(w["g"] @ h)
    o = np.zeros((H, dv))
    for i in range(H):
        g = i // (H // G)
        y = attention_weights(q[i], K[:, g], c["scale"]) @ V[:, g]
        o[i] = gate[i] * rotate_pairs(y, -pos, rot["base"], dv)
    return w["o"] @ o.reshape(-1) + w["o.b"]


# ---------------------------------------------------------------------------------------------------- minimal gated recurrence
def mingru_candidate(u):
    return np.where(u >= 0, u + 0.5, sigmoid(u))


def mingru_step(w, c, h, st):
    z, u = sigmoid(w["z"] @ h + w["z.b"]), w["x"] @ h + w["x.b"]
    st["S"] = (1.0 - z) * st["S"] + z * mingru_candidate(u)
    return w["o"] @ (st["S"] * silu(w["g"] @ h))


MIXERS = {"attention": attention_step, "mingru": mingru_step}


def new_state(entry, width, taps):
    st = {"conv": np.zeros((taps - 1, width))}
    if entry["type"] == "attention":
        return {**st, "k": [], "v": []}
    return {**st, "S": np.zeros(entry["mixer"]["width"])}


# ---------------------------------------------------------------------------------------------------- feed-forward
def dense_ff(w, h):
    return w["down"] @ (np.maximum(w["gate"] @ h, 0.0) * (w["up"] @ h))


def expert_ff(up, down, h):
    return down @ np.square(np.maximum(up @ h, 0.0))


def route(z, correction, top):
    """Which outputs of the router are chosen, and their weights."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    chosen = np.argsort(-(s + correction), kind="stable")[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20)


def moe_ff(w, c, h):
    r = c["router"]
    y = np.zeros(len(h))
    for e, p in zip(*route(w["router"] @ h, w["correction"], r["top"])):
        y += p * (h if e >= r["experts"] else expert_ff(w[f"e{e}.up"], w[f"e{e}.down"], h))
    if c.get("shared"):
        y += sigmoid(w["shared.sg"] @ h)[0] * expert_ff(w["shared.up"], w["shared.down"], h)
    return y


def feed_forward(w, c, h):
    return dense_ff(w, h) if c["kind"] == "dense" else moe_ff(w, c, h)


# ---------------------------------------------------------------------------------------------------- the whole model
def layer_runs(cfg):
    """(layer, pass that begins here or None) of every layer run, in order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    passes = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + passes + [(i, None) for i in range(b, n)]


class Oracle:
    def __init__(self, cfg: dict, tensors: dict):
        self.cfg, self.t = cfg, {k: np.asarray(v, F) for k, v in tensors.items()}
        self.runs = layer_runs(cfg)
        self.w = [self.sub(f"l{i}.") for i in range(len(cfg["layers"]))]
        self.reset()

    def sub(self, prefix, of=None):
        return {k[len(prefix):]: v for k, v in (of or self.t).items() if k.startswith(prefix)}

    def reset(self):
        self.state = [new_state(self.cfg["layers"][i], self.cfg["width"], self.cfg["canon"]["taps"]) for i, _ in self.runs]
        self.trace = []

    def layer(self, i, x, st):
        e, w, eps = self.cfg["layers"][i], self.w[i], self.cfg["norm"]["eps"]
        h = rms_norm(x, eps, w["norm1"])
        add, st["conv"] = causal_conv(w["canon1"], h, st["conv"])
        y = MIXERS[e["type"]](self.sub("mix.", w), e["mixer"], h + add, st)
        x = x + rms_norm(y, eps, w["norm1b"]) * w["ls1"]
        if e.get("mlp"):
            y = feed_forward(self.sub("mlp.", w), e["mlp"], rms_norm(x, eps, w["norm2"]))
            x = x + rms_norm(y, eps, w["norm2b"]) * w["ls2"]
        return x

    def token(self, tok, keep_layers=False):
        x0 = self.t["embed"][tok].copy()
        x = x0
        for (i, begins), st in zip(self.runs, self.state):
            if begins is not None:
                x = self.t["loop.in"] @ np.concatenate([x, x0]) + self.t["loop.step"][begins]
            x = self.layer(i, x, st)
            if keep_layers:
                self.trace.append(x.copy())
        return self.t["head"] @ rms_norm(x, self.cfg["norm"]["eps"], self.t["final.norm"])

    def run(self, ids):
        return np.array([self.token(t) for t in ids])

    def greedy(self, prompt, n):
        self.reset()
        logits = self.run(prompt)[-1]
        out = []
        for _ in range(n):
            out.append(int(np.argmax(logits)))
            if len(out) < n:
                logits = self.token(out[-1])
        return out
