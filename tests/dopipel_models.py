"""Small random Dopipel models for the tests, with weights scaled so that mistakes show: attention is peaked (single keys
matter), gates and layer scales are far from neutral, recurrences span fast and slow channels, corrections change choices."""
from __future__ import annotations

import math

import numpy as np

from dopipel_oracle import Oracle
from hybrid_oracle import write_model


def attention(heads, kv_heads, dim, vdim, rot, base=10000.0, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                           "rot": {"base": base, "dims": rot}, "scale": scale or 1.2 / math.sqrt(dim)}}


def mingru(width):
    return {"type": "mingru", "mixer": {"width": width}}


def dense(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def moe(layer, experts, top, ff, identity=0, shared=0):
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top, "identity": identity}, "expert": {"ff": ff}}
    return {**layer, "mlp": {**mlp, "shared": {"ff": shared}} if shared else mlp}


def bare(layer):
    return {**layer, "mlp": None}


def config(width, vocab, layers, taps=3, loop=None, eps=2e-5):
    cfg = {"architecture": "Dopipel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}
    return {**cfg, "loop": dict(zip(("start", "stop", "times"), loop))} if loop else cfg


CONFIGS = {
    # every part; the loop covers a mixture and both mixers
    "mixed": config(96, 333, [dense(attention(6, 2, 40, 24, 24), 88), moe(mingru(72), 10, 3, 40, identity=3, shared=56),
                              moe(attention(4, 4, 16, 32, 16, base=700.0), 6, 2, 24, shared=32), dense(mingru(104), 56)], loop=(1, 3, 2)),
    # sizes that are not multiples of 8, a loop over everything, a long convolution, a layer without feed-forward, no rotated keys
    "odd": config(52, 77, [moe(attention(5, 1, 20, 12, 10, base=500.0), 7, 2, 18, identity=1, shared=10), bare(mingru(36)),
                           dense(attention(3, 3, 11, 14, 0), 30), moe(bare(mingru(21)), 3, 1, 9)], taps=5, loop=(0, 4, 2), eps=1e-3),
    # no loop, a convolution of the token itself only, one head, every output of the router chosen
    "plain": config(64, 90, [dense(attention(1, 1, 8, 40, 8), 24), moe(mingru(40), 3, 4, 16, identity=1)], taps=1),
    # many query heads per key/value head, wide heads, the first layers alone ahead of the loop, only identity experts beside one
    "heads": config(160, 200, [dense(attention(20, 1, 16, 8, 12), 48), bare(attention(3, 3, 136, 72, 64)),
                               moe(attention(8, 2, 64, 128, 32), 1, 2, 40, identity=5, shared=8)], taps=4, loop=(2, 3, 2)),
}


def weights(cfg, seed, decided=False):
    """decided: corrections so far apart that they alone choose the experts, so that a rounded logit cannot change a choice."""
    rng = np.random.default_rng(seed)
    W, t = cfg["width"], {}
    mat = lambda n, k, gain=1.0: rng.standard_normal((n, k)) * gain / math.sqrt(k)
    vec = lambda n, lo, hi: rng.uniform(lo, hi, n)
    t["embed"] = rng.standard_normal((cfg["vocab"], W))
    if cfg.get("loop"):
        t["loop.in"] = mat(W, 2 * W, 1.2)
        t["loop.step"] = rng.standard_normal((cfg["loop"]["times"], W))
    for i, e in enumerate(cfg["layers"]):
        p, c = f"l{i}.", e["mixer"]
        m = p + "mix."
        t[p + "canon1"] = rng.standard_normal((W, cfg["canon"]["taps"])) * 0.6
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if e.get("mlp") else ()):
            t[p + n] = vec(W, 0.5, 1.5)
        for n in ("ls1",) + (("ls2",) if e.get("mlp") else ()):
            t[p + n] = vec(W, 0.3, 1.2)
        if e["type"] == "attention":
            H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
            for n, rows, gain in (("q", H * d, 1.6), ("k", G * d, 1.6), ("v", G * dv, 1.0)):
                t[m + n], t[m + n + ".b"] = mat(rows, W, gain), vec(rows, -0.5, 0.5)
            t[m + "g"] = mat(H, W, 1.5)
            t[m + "o"], t[m + "o.b"] = mat(W, H * dv), vec(W, -0.3, 0.3)
        else:
            n = c["width"]
            t[m + "z"], t[m + "z.b"] = mat(n, W), vec(n, -6.0, 1.0)
            t[m + "x"], t[m + "x.b"] = mat(n, W, 1.5), vec(n, -1.0, 1.0)
            t[m + "g"], t[m + "o"] = mat(n, W, 1.5), mat(W, n)
        f = e.get("mlp")
        if f and f["kind"] == "dense":
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(f["ff"], W, 1.5), mat(f["ff"], W), mat(W, f["ff"])
        elif f:
            r = f["router"]
            outputs = r["experts"] + r["identity"]
            t[p + "mlp.router"], t[p + "mlp.correction"] = mat(outputs, W, 1.5), vec(outputs, -0.1, 0.1)
            if decided:
                t[p + "mlp.correction"] = 2.0 * rng.permutation(outputs)
            for k in range(r["experts"]):
                t[p + f"mlp.e{k}.up"], t[p + f"mlp.e{k}.down"] = mat(f["expert"]["ff"], W), mat(W, f["expert"]["ff"])
            if f.get("shared"):
                s = f["shared"]["ff"]
                t[p + "mlp.shared.up"], t[p + "mlp.shared.down"] = mat(s, W), mat(W, s)
                t[p + "mlp.shared.sg"] = mat(1, W, 1.5)
    t["final.norm"] = vec(W, 0.5, 1.5)
    t["head"] = mat(cfg["vocab"], W, 2.0)
    return t


def build(folder, name, seed=1, decided=False):
    """Writes the model folder and returns (configuration, oracle over the tensors as stored)."""
    cfg = CONFIGS[name]
    return cfg, Oracle(cfg, write_model(folder, cfg, weights(cfg, seed, decided)))
