"""Plain implementation of the hybrid decoder's mechanisms (architecture "Fazilorn"): test infrastructure.

Everything runs token by token in float64 on numpy arrays, one function per mechanism, with explicit state, so that a cut
of the sequence anywhere is the same computation.  Nothing here is shared with the product path.

  x : residual row        h : normalised row        W[out, in] linears applied as W @ h
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np

F = np.float64


# ---------------------------------------------------------------------------------------------------- elementwise pieces
def sigmoid(z):
    z = np.asarray(z, F)
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, eps, weight=None):
    """x / sqrt(mean(x^2) + eps), times a weight when there is one; over the last axis."""
    y = x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def rotate_pairs(x, pos, base, dims):
    """Rotation of the first `dims` entries of the last axis in neighbouring pairs (2i, 2i+1) by pos * base^(-2i/dims)."""
    y = np.array(x, F)
    i = np.arange(dims // 2)
    a = pos * np.power(F(base), -2.0 * i / dims)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * np.cos(a) - v * np.sin(a)
    y[..., 1:dims:2] = v * np.cos(a) + u * np.sin(a)
    return y


def swiglu(w, h):
    return w["down"] @ (silu(w["gate"] @ h) * (w["up"] @ h))


# ---------------------------------------------------------------------------------------------------- recurrent mixers
def gla_decay(z, tau):
    """Per-channel decay sigmoid(z)^(1/tau), through the logarithm of the sigmoid."""
    return np.exp(-np.logaddexp(0.0, -z) / tau)


def gla_state_step(S, q, k, v, alpha):
    """One head: S[dim, vdim] <- diag(alpha) S + k v^T, read with q after the update."""
    S = alpha[:, None] * S + np.outer(k, v)
    return S, S.T @ q


def wkv_state_step(S, r, k, v, u, w):
    """One head: the read sees the old state plus the current pair weighted by u; the decay w acts afterwards."""
    o = (S + np.outer(u * k, v)).T @ r
    return w[:, None] * S + np.outer(k, v), o


def gla_step(w, c, eps, h, st):
    H, d, dv = c["heads"], c["dim"], c["vdim"]
    q = (w["q"] @ h).reshape(H, d) * d ** -0.5
    k = (w["k"] @ h).reshape(H, d)
    v = (w["v"] @ h).reshape(H, dv)
    alpha = gla_decay(w["a2"] @ (w["a1"] @ h) + w["a2.b"], c["tau"]).reshape(H, d)
    o = np.zeros((H, dv))
    for i in range(H):
        st["S"][i], o[i] = gla_state_step(st["S"][i], q[i], k[i], v[i], alpha[i])
    o = rms_norm(o, eps, w["norm"]).reshape(-1)
    return w["o"] @ (o * silu(w["g"] @ h))


def wkv_step(w, c, eps, h, st):
    H, d = c["heads"], c["dim"]
    mix = {n: h + (st["prev"] - h) * w["mu." + n] for n in "rkvgw"}
    st["prev"] = h.copy()
    r, k, v = ((w[n] @ mix[n]).reshape(H, d) for n in "rkv")
    gate = silu(w["g"] @ mix["g"])
    decay = np.exp(-np.exp(w["w2"] @ np.tanh(w["w1"] @ mix["w"]) + w["w0"])).reshape(H, d)
    o = np.zeros((H, d))
    for i in range(H):
        st["S"][i], o[i] = wkv_state_step(st["S"][i], r[i], k[i], v[i], w["u"][i], decay[i])
    return w["o"] @ (rms_norm(o, eps).reshape(-1) * w["norm"] * gate)


# ---------------------------------------------------------------------------------------------------- latent attention
def softmax_with_sink(scores, sink):
    m = max(scores.max(), sink)
    p = np.exp(scores - m)
    return p / (p.sum() + np.exp(sink - m))


def latent_attention_step(w, c, eps, h, st):
    H, d, rd, dv, R = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    pos = len(st["c"])
    rot = c["rot"]
    q = (w["uq"] @ rms_norm(w["dq"] @ h, eps, w["dq.norm"])).reshape(H, d + rd)
    low = w["dkv"] @ h
    st["c"].append(rms_norm(low[:R], eps, w["dkv.norm"]))
    st["kr"].append(rotate_pairs(low[R:], pos, rot["base"], rot["dims"]))
    first = max(0, pos - c["mask"]["size"] + 1)
    C, KR = np.array(st["c"][first:]), np.array(st["kr"][first:])
    o = np.zeros((H, dv))
    for i in range(H):
        K = C @ w["uk"][i * d:(i + 1) * d].T
        V = C @ w["uv"][i * dv:(i + 1) * dv].T
        s = (K @ q[i, :d] + KR @ rotate_pairs(q[i, d:], pos, rot["base"], rot["dims"])) * c["scale"]
        o[i] = softmax_with_sink(s, w["sink"][i]) @ V
    return w["o"] @ (o.reshape(-1) * sigmoid(w["g"] @ h))


MIXERS = {"gla": gla_step, "wkv": wkv_step, "latent_attention": latent_attention_step}


def new_state(entry, width):
    c = entry["mixer"]
    if entry["type"] == "gla":
        return {"S": np.zeros((c["heads"], c["dim"], c["vdim"]))}
    if entry["type"] == "wkv":
        return {"S": np.zeros((c["heads"], c["dim"], c["dim"])), "prev": np.zeros(width)}
    return {"c": [], "kr": []}


# ---------------------------------------------------------------------------------------------------- the whole model
class Oracle:
    def __init__(self, cfg: dict, tensors: dict):
        self.cfg, self.t = cfg, {k: np.asarray(v, F) for k, v in tensors.items()}
        self.reset()

    def reset(self):
        self.state = [new_state(e, self.cfg["width"]) for e in self.cfg["layers"]]
        self.trace = []

    def owner(self, i):
        while self.cfg["layers"][i].get("weights_of") is not None:
            i = self.cfg["layers"][i]["weights_of"]
        return i

    def sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def token(self, tok, keep_layers=False):
        eps = self.cfg["norm"]["eps"]
        x = self.t["embed"][tok].copy()
        for i, e in enumerate(self.cfg["layers"]):
            p = f"l{self.owner(i)}."
            h = rms_norm(x, eps, self.t[p + "norm1"])
            y = MIXERS[e["type"]](self.sub(p + "mix."), e["mixer"], eps, h, self.state[i])
            if e.get("mlp"):
                y = y + swiglu(self.sub(p + "mlp."), h)
            x = x + y
            if keep_layers:
                self.trace.append(x.copy())
        logits = self.t["head"] @ rms_norm(x, eps, self.t["final.norm"])
        cap = self.cfg.get("logit_softcap")
        return logits if not cap else cap * np.tanh(logits / cap)

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


# ---------------------------------------------------------------------------------------------------- model folders
def bf16_bits(a):
    """fp32 -> bf16 bit patterns, round to nearest even."""
    b = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((b + 0x7FFF + ((b >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_values(bits):
    return (bits.astype(np.uint32) << 16).view(np.float32)


def write_model(folder, cfg, tensors):
    """config.json + model.safetensors (bf16); returns the tensors as stored."""
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    head, blobs, off, stored = {}, [], 0, {}
    for name, a in tensors.items():
        bits = bf16_bits(a)
        stored[name] = bf16_values(bits).astype(F)
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [off, off + bits.nbytes]}
        off += bits.nbytes
        blobs.append(bits.tobytes())
    raw = json.dumps(head).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(raw)) + raw + b"".join(blobs))
    return stored


def read_tensors(path):
    raw = Path(path).read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    head, data, out = json.loads(raw[8:8 + n]), raw[8 + n:], {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        a, b = t["data_offsets"]
        out[name] = bf16_values(np.frombuffer(data[a:b], np.uint16)).reshape(t["shape"]).astype(F)
    return out
