"""Small random models of the hybrid architecture for the tests, with weights scaled so that mistakes show: attention is peaked
(single keys matter), sinks and gates are far from neutral, decays span fast and slow channels."""
from __future__ import annotations

import math

import numpy as np

from hybrid_oracle import Oracle, write_model


def gla(heads, dim, vdim, tau, ff):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": ff and {"kind": "dense", "ff": ff}}


def wkv(heads, dim, ff):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": ff and {"kind": "dense", "ff": ff}}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, ff, base=10000.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim},
                      "scale": scale or 1 / math.sqrt(dim + rot_dim)},
            "mlp": ff and {"kind": "dense", "ff": ff}}


def again(entry, of):
    return {**entry, "weights_of": of}


def config(width, vocab, layers, eps=2e-5, softcap=25.0):
    return {"architecture": "Fazilorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": softcap, "layers": layers}


def _mixed():
    a, b, c = gla(3, 24, 40, 8.0, 88), wkv(5, 16, 120), latent(3, 24, 8, 32, 40, 48, 21, 72)
    return config(96, 333, [a, b, c, again(c, 2), again(b, 1), again(a, 0)])


CONFIGS = {
    # every mixer, shared weights in another order than the owners
    "mixed": _mixed(),
    # sizes that are not multiples of 8, one head, no feed-forward in places, no cap
    "odd": config(52, 77, [latent(1, 10, 4, 12, 22, 18, 9, None, base=500.0), wkv(3, 12, 30), gla(1, 12, 20, 1.0, None),
                           latent(5, 6, 2, 10, 14, 30, 1, 26)], eps=1e-3, softcap=None),
    # attention first and last, windows around the tile sizes of the kernels, wide value heads
    "windows": config(128, 256, [latent(9, 16, 16, 72, 64, 72, 64, 96), latent(2, 40, 24, 96, 32, 128, 17, None),
                                 gla(2, 64, 128, 32.0, 64), latent(4, 32, 8, 48, 48, 32, 100, 64)], softcap=5.0),
    # head sizes beyond 64 in the recurrences
    "wide_heads": config(160, 200, [wkv(2, 80, 48), gla(1, 160, 72, 16.0, 40), gla(2, 128, 24, 4.0, 24)]),
}


def weights(cfg, seed):
    """Random tensors for a configuration; the residual stream grows like that of a trained model (unit-size rows)."""
    rng = np.random.default_rng(seed)
    W, t = cfg["width"], {}
    mat = lambda n, k, gain=1.0: rng.standard_normal((n, k)) * gain / math.sqrt(k)
    vec = lambda n, lo, hi: rng.uniform(lo, hi, n)
    t["embed"] = rng.standard_normal((cfg["vocab"], W))
    for i, e in enumerate(cfg["layers"]):
        if e.get("weights_of") is not None:
            continue
        p, c = f"l{i}.", e["mixer"]
        m = p + "mix."
        H, d = c["heads"], c["dim"]
        dv = c.get("vdim", d)
        t[p + "norm1"] = vec(W, 0.5, 1.5)
        t[m + "g"] = mat(H * dv, W, 1.5)
        t[m + "o"] = mat(W, H * dv, 0.8)
        if e["type"] in ("gla", "wkv"):
            rank = int(rng.integers(3, 20))
            q, a, b, bias = ("q", "a1", "a2", "a2.b") if e["type"] == "gla" else ("r", "w1", "w2", "w0")
            t[m + q], t[m + "k"], t[m + "v"] = mat(H * d, W), mat(H * d, W), mat(H * dv, W)
            t[m + a], t[m + b] = mat(rank, W), mat(H * d, rank)
            t[m + bias] = vec(H * d, -1.0, 4.0) if e["type"] == "gla" else vec(H * d, -5.0, 0.5)
        if e["type"] == "gla":
            t[m + "norm"] = vec(dv, 0.5, 1.5)
        if e["type"] == "wkv":
            t[m + "norm"] = vec(H * d, 0.5, 1.5)
            t[m + "u"] = vec(H * d, -1.0, 2.0).reshape(H, d)
            for n in "rkvgw":
                t[m + "mu." + n] = vec(W, 0.0, 1.0)
        if e["type"] == "latent_attention":
            R, rd, qr = c["kv_rank"], c["rot_dim"], c["q_rank"]
            t[m + "dq"], t[m + "dq.norm"] = mat(qr, W), vec(qr, 0.5, 1.5)
            uq = mat(H * (d + rd), qr, 2.5).reshape(H, d + rd, qr)
            uq[:, d:] *= 2.0                     # the rotated part weighs as much as the rest
            t[m + "uq"] = uq.reshape(-1, qr)
            t[m + "dkv"], t[m + "dkv.norm"] = mat(R + rd, W), vec(R, 0.5, 1.5)
            t[m + "uk"], t[m + "uv"] = mat(H * d, R, 2.0), mat(H * dv, R, 2.0)
            t[m + "sink"] = vec(H, 2.0, 7.0)
        if e.get("mlp"):
            ff = e["mlp"]["ff"]
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(ff, W, 1.5), mat(ff, W), mat(W, ff, 0.8)
    t["final.norm"] = vec(W, 0.5, 1.5)
    t["head"] = mat(cfg["vocab"], W, 2.0)
    return t


def build(folder, name, seed=1):
    """Writes the model folder and returns (configuration, oracle over the tensors as stored)."""
    cfg = CONFIGS[name]
    return cfg, Oracle(cfg, write_model(folder, cfg, weights(cfg, seed)))


def prompt(cfg, n, seed):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n).astype(np.int32)


def rows_error(got, want):
    """Worst row: rms difference of the mean-free logits over their rms size."""
    g, w = got - got.mean(-1, keepdims=True), want - want.mean(-1, keepdims=True)
    return float((np.sqrt(np.mean((g - w) ** 2, -1)) / np.sqrt(np.mean(w * w))).max())
