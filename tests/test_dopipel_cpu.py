"""Dopipel models without a GPU: configuration and checkpoint errors, the registry, closed forms of the oracle's pieces, and what
the test weights can tell apart (a mistake planted in the oracle must move the logits by far more than any tolerance)."""
import copy
import ctypes as C
import json

import numpy as np
import pytest

import dopipel_oracle as do
import hybrid_oracle as ho
from dopipel_models import CONFIGS, attention, bare, build, config, dense, mingru, moe, weights
from hybrid_models import prompt, rows_error


def check(libs, cfg):
    h, n = libs.host(), C.c_size_t(0)
    rc = h.dh_hybrid_check_config(json.dumps(cfg).encode(), C.byref(n))
    return n.value if rc == 0 else h.dh_last_error().decode()


def test_configurations_are_read(libs):
    for name, cfg in CONFIGS.items():
        assert check(libs, cfg) == len(cfg["layers"]), name
    one = lambda e, **kw: check(libs, config(64, 50, [e], **kw))
    ok = dense(attention(4, 2, 16, 8, 8), 32)
    assert one(ok) == 1
    assert "unknown mixer" in one({**ok, "type": "gla"})
    assert "multiple of 'kv_heads'" in one(dense(attention(4, 3, 16, 8, 8), 32))
    assert "rot.dims" in one(dense(attention(4, 2, 16, 8, 7), 32))
    assert "rot.dims" in one(dense(attention(4, 2, 16, 8, 18), 32))
    assert "vdim" in one(dense(attention(4, 2, 16, 7, 8), 32))
    assert "width" in one(bare(mingru(0)))
    assert "'ff'" in one(dense(mingru(8), 0))
    assert "unknown feed-forward" in one({**bare(mingru(8)), "mlp": {"kind": "glu", "ff": 8}})
    assert "router.top" in one(moe(mingru(8), 4, 6, 8, identity=1))
    assert "experts" in one(moe(mingru(8), 0, 1, 8, identity=1))
    assert "outputs" in one(moe(mingru(8), 1020, 1, 8, identity=5))
    assert "taps" in one(ok, taps=17) and "taps" in one(ok, taps=0)
    assert "loop" in one(ok, loop=(0, 2, 1)) and "loop" in one(ok, loop=(1, 1, 1)) and "loop" in one(ok, loop=(0, 1, 0))
    assert "vocab" in check(libs, config(64, 0, [ok]))


def test_registry_and_missing_tensors(libs, ref_backend, tmp_path):
    h = libs.host()
    buf = C.create_string_buffer(256)
    assert h.dh_architectures(buf, 256) == 0 and "Dopipel" in buf.value.decode().split()

    def opened(path, cfg, t):
        ho.write_model(path, cfg, t)
        m = h.dh_model_open(ref_backend, str(path).encode(), libs.DET_F32, 32, 8)
        if not m:
            return h.dh_last_error().decode()
        h.dh_model_free(m)
        return None

    for name, cfg in CONFIGS.items():
        assert opened(tmp_path / name, cfg, weights(cfg, 1)) is None
    cfg = CONFIGS["mixed"]
    for tensor in ("loop.in", "loop.step", "l0.canon1", "l0.mix.k.b", "l1.mlp.e9.down", "l1.mlp.correction", "l2.mlp.shared.sg", "l3.ls2"):
        t = weights(cfg, 1)
        del t[tensor]
        assert tensor in opened(tmp_path / "missing", cfg, t)
    t = weights(cfg, 1)
    t["l1.mlp.router"] = t["l1.mlp.router"][:-1]
    assert "l1.mlp.router" in opened(tmp_path / "shape", cfg, t)


def test_oracle_pieces():
    add, past = do.causal_conv(np.array([[1.0, 10.0, 100.0]]), np.array([3.0]), np.array([[1.0], [2.0]]))
    assert add == 321.0 and past.tolist() == [[2.0], [3.0]]
    chosen, w = do.route(np.log(np.array([0.5, 0.3, 0.2])), np.array([-1.0, 0.0, 0.2]), 2)
    assert chosen.tolist() == [2, 1] and np.allclose(w, [0.4, 0.6])
    assert np.allclose(do.mingru_candidate(np.array([-1e-12, 0.0, 2.0])), [0.5, 0.5, 2.5])
    assert do.layer_runs(config(8, 8, [bare(mingru(8))] * 4, loop=(1, 3, 2))) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    # attention of one key gives its value back whatever the position: the rotation of the values is undone
    w = {n: np.zeros(s) for n, s in (("q", (2, 3)), ("k", (2, 3)), ("v", (4, 3)), ("g", (1, 3)))}
    w.update({"q.b": np.zeros(2), "k.b": np.array([0.0, 0.0]), "v.b": np.arange(4.0), "o": np.eye(4), "o.b": np.zeros(4)})
    c = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 4, "rot": {"base": 10.0, "dims": 2}, "scale": 1.0}
    w["k.b"], w["q.b"] = np.array([60.0, 0.0]), np.array([60.0, 0.0])
    st = {"k": [], "v": []}
    for _ in range(5):      # aligned q and k: the token itself takes all the weight
        assert np.allclose(do.attention_step(w, c, np.zeros(3), st), 0.5 * np.arange(4.0))


def changed(change):
    """A run over a changed model: change(cfg, tensors) in place."""
    def run(cfg, tensors, ids):
        cfg, tensors = copy.deepcopy(cfg), dict(tensors)
        change(cfg, tensors)
        return do.Oracle(cfg, tensors).run(ids)
    return run


def patched(**kw):
    def run(cfg, tensors, ids):
        with pytest.MonkeyPatch.context() as m:
            for name, fn in kw.items():
                if name in do.MIXERS:
                    m.setitem(do.MIXERS, name, fn)
                else:
                    m.setattr(do, name, fn)
            return do.Oracle(cfg, tensors).run(ids)
    return run


def _each_layer(fn):
    def change(cfg, t):
        for i, e in enumerate(cfg["layers"]):
            fn(f"l{i}.", e, cfg, t)
    return change


def _zero(*names):
    def fn(p, e, cfg, t):
        for n in names:
            if p + n in t:
                t[p + n] = np.zeros_like(t[p + n])
    return changed(_each_layer(fn))


def _no_shift(p, e, cfg, t):
    t[p + "canon1"] = np.roll(t[p + "canon1"], 1, axis=1)


def _groups(p, e, cfg, t):
    if e["type"] == "attention" and e["mixer"]["kv_heads"] > 1:
        for n in ("k", "v"):
            G = e["mixer"]["kv_heads"]
            for b in ("", ".b"):
                a = t[p + f"mix.{n}{b}"]
                t[p + f"mix.{n}{b}"] = np.roll(a.reshape(G, -1), 1, axis=0).reshape(a.shape)


def _base(p, e, cfg, t):
    if e["type"] == "attention":
        e["mixer"]["rot"]["base"] *= 1.3


def _no_value_rotation(w, c, h, st, orig=do.attention_step, rot=do.rotate_pairs):
    dv = c["vdim"]
    with pytest.MonkeyPatch.context() as m:
        m.setattr(do, "rotate_pairs", lambda x, pos, base, dims: x if x.shape[-1] == dv and dims == dv else rot(x, pos, base, dims))
        return orig(w, c, h, st)


def _lost_state(w, c, h, st, orig=do.mingru_step):
    st["n"] = st.get("n", 0) + 1
    if st["n"] == 30:
        st["S"] = np.zeros_like(st["S"])
    return orig(w, c, h, st)


def _first_key_lost(q, K, scale, orig=do.attention_weights):
    p = orig(q, K, scale)
    if len(p) > 40:
        p[0] = 0.0
        p /= p.sum()
    return p


def _no_identity(z, correction, top, orig=do.route):
    chosen, w = orig(z, correction, top)
    return chosen, np.where(chosen >= 10, 0.0, w) if len(z) == 13 else w


def _weights_with_correction(z, correction, top, orig=do.route):
    chosen, _ = orig(z, correction, top)
    s = np.exp(z - z.max())
    s = s / s.sum() + correction
    return chosen, s[chosen] / s[chosen].sum()


def _shared_state(cfg, tensors, ids):
    o = do.Oracle(cfg, tensors)
    o.state[3], o.state[4] = o.state[1], o.state[2]       # both passes of the loop on one state
    return o.run(ids)


MISTAKES = {
    "no convolution": _zero("canon1"), "taps shifted": changed(_each_layer(_no_shift)), "no projection bias": _zero("mix.q.b", "mix.k.b", "mix.v.b"),
    "no output bias": _zero("mix.o.b"), "no step vector": changed(lambda cfg, t: t.update({"loop.step": t["loop.step"] * 0})),
    "no embedding in the loop": changed(lambda cfg, t: t.update({"loop.in": np.hstack([t["loop.in"][:, :96], t["loop.in"][:, 96:] * 0])})),
    "one pass": changed(lambda cfg, t: cfg["loop"].update(times=1)), "passes share a state": _shared_state,
    "wrong group": changed(_each_layer(_groups)), "rotation base": changed(_each_layer(_base)),
    "values not rotated": patched(attention=_no_value_rotation), "state lost": patched(mingru=_lost_state),
    "first key lost": patched(attention_weights=_first_key_lost), "identity experts dropped": patched(route=_no_identity),
    "no correction": _zero("mlp.correction"), "correction in the weights": patched(route=_weights_with_correction),
    "no shared gate": _zero("mlp.shared.sg"), "no output gate": _zero("mix.g"),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_planted_mistakes_show(name, tmp_path):
    cfg, oracle = build(tmp_path, "mixed")
    ids = prompt(cfg, 60, 3)
    want = oracle.run(ids)
    tensors = {k: v for k, v in oracle.t.items()}
    got = MISTAKES[name](cfg, tensors, ids)
    assert rows_error(got[40:], want[40:]) > 0.02          # 200 times the 32-bit tolerance
