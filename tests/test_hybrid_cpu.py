"""Hybrid models without a GPU: configuration and checkpoint errors, the registry, and what the oracle's test weights can tell
apart (a mistake planted in the oracle must move the logits by far more than any tolerance the GPU tests use)."""
import ctypes as C
import json
import struct

import numpy as np
import pytest

import hybrid_oracle as ho
from hybrid_models import CONFIGS, build, config, gla, latent, prompt, rows_error, weights, wkv
from hybrid_oracle import Oracle


def check(libs, cfg):
    h, n = libs.host(), C.c_size_t(0)
    rc = h.dh_hybrid_check_config(json.dumps(cfg).encode(), C.byref(n))
    return n.value if rc == 0 else h.dh_last_error().decode()


def test_configurations_are_read(libs):
    for name, cfg in CONFIGS.items():
        assert check(libs, cfg) == len(cfg["layers"]), name
    bad = lambda **kw: check(libs, {**config(64, 50, [gla(2, 16, 16, 4.0, 32)]), **kw})
    assert "vocab" in bad(vocab=0)
    assert "layers" in bad(layers=[])
    layer = lambda e: check(libs, config(64, 50, [e]))
    assert "unknown mixer" in layer({"type": "conv", "mixer": {"heads": 1, "dim": 8}})
    assert "unknown feed-forward" in layer({**wkv(2, 8, None), "mlp": {"kind": "routed", "ff": 8}})
    assert "tau" in layer(gla(1, 8, 8, 0.0, None))
    assert "mask.size" in layer(latent(1, 8, 4, 8, 8, 8, 0, None))
    e = latent(1, 8, 4, 8, 8, 8, 4, None)
    e["mixer"]["rot"]["dims"] = 6
    assert "rot.dims" in layer(e)
    two = lambda e: check(libs, config(64, 50, [gla(2, 16, 16, 4.0, 32), e]))
    assert two({**gla(2, 16, 16, 4.0, 32), "weights_of": 0}) == 2
    assert "other sizes" in two({**gla(2, 16, 24, 4.0, 32), "weights_of": 0})
    assert "names no layer" in two({**gla(2, 16, 16, 4.0, 32), "weights_of": 2})
    assert "circle" in check(libs, config(64, 50, [{**gla(2, 16, 16, 4.0, 32), "weights_of": 1}, {**gla(2, 16, 16, 4.0, 32), "weights_of": 0}]))


def test_registry_names_and_open_errors(libs, ref_backend, tmp_path):
    h = libs.host()
    buf = C.create_string_buffer(256)
    assert h.dh_architectures(buf, 256) == 0
    assert {"qwen35", "Fazilorn"} <= set(buf.value.decode().split())

    def opened(path):
        m = h.dh_model_open(ref_backend, str(path).encode(), libs.DET_F32, 32, 8)
        if m:
            h.dh_model_free(m)
            return None
        return h.dh_last_error().decode()

    assert "no such" in opened(tmp_path / "absent")
    cfg = CONFIGS["odd"]
    ho.write_model(tmp_path / "good", cfg, weights(cfg, 1))
    assert opened(tmp_path / "good") is None            # loading needs buffers only
    ho.write_model(tmp_path / "arch", {**cfg, "architecture": "Other"}, weights(cfg, 1))
    assert "Other" in opened(tmp_path / "arch")
    t = weights(cfg, 1)
    del t["l1.mix.w0"]
    ho.write_model(tmp_path / "missing", cfg, t)
    assert "l1.mix.w0" in opened(tmp_path / "missing")
    t = weights(cfg, 1)
    t["l0.mix.uk"] = t["l0.mix.uk"][:-1]
    ho.write_model(tmp_path / "shape", cfg, t)
    assert "l0.mix.uk" in opened(tmp_path / "shape")
    t = weights(cfg, 1)
    t["head"][3, 5] = np.inf
    ho.write_model(tmp_path / "inf", cfg, t)
    assert "not finite" in opened(tmp_path / "inf")


@pytest.mark.parametrize("damage,word", [("header", "header"), ("offsets", "offsets"), ("size", "disagree"), ("json", "JSON")])
def test_damaged_safetensors(damage, word, libs, ref_backend, tmp_path):
    h, cfg = libs.host(), CONFIGS["odd"]
    ho.write_model(tmp_path, cfg, weights(cfg, 1))
    f = tmp_path / "model.safetensors"
    raw = f.read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    head, data = json.loads(raw[8:8 + n]), raw[8 + n:]
    if damage == "header":
        f.write_bytes(struct.pack("<Q", 1 << 40) + raw[8:])
    else:
        if damage == "offsets":
            head["head"]["data_offsets"][1] += 1 << 30
        if damage == "size":
            head["head"]["shape"][0] -= 1
        text = json.dumps(head).encode()
        if damage == "json":
            text = text[:-1]
        f.write_bytes(struct.pack("<Q", len(text)) + text + data)
    assert not h.dh_model_open(ref_backend, str(tmp_path).encode(), libs.DET_F32, 32, 8)
    assert word in h.dh_last_error().decode()


def test_a_backend_without_float_ops_says_so(libs, ref_backend, tmp_path):
    h, cfg = libs.host(), CONFIGS["odd"]
    ho.write_model(tmp_path, cfg, weights(cfg, 1))
    m = h.dh_model_open(ref_backend, str(tmp_path).encode(), libs.DET_F32, 32, 8)
    assert m
    ids = np.zeros(4, np.int32)
    assert h.dh_model_forward(m, ids.ctypes.data, 4) != 0
    assert "floating-point" in h.dh_last_error().decode()
    ids[2] = cfg["vocab"]
    assert h.dh_model_forward(m, ids.ctypes.data, 4) != 0 and "outside the embedding" in h.dh_last_error().decode()
    h.dh_model_free(m)


def _latent_with(change):
    """latent_attention_step of a changed layer description."""
    def step(w, c, eps, h, st, orig=ho.latent_attention_step):
        w, c = dict(w), json.loads(json.dumps(c))
        change(w, c)
        return orig(w, c, eps, h, st)
    return step


def _bump_window(by):
    def change(w, c):
        c["mask"]["size"] = max(1, c["mask"]["size"] + by)
    return _latent_with(change)


def _no_sink(w, c):
    w["sink"] = np.full_like(w["sink"], -1e30)


def _base(w, c):
    c["rot"]["base"] *= 1.5


def _no_shift(w, c, eps, h, st, orig=ho.wkv_step):
    st["prev"] = h.copy()
    return orig(w, c, eps, h, st)


def _read_first(w, c, eps, h, st, orig=ho.wkv_step):
    w = dict(w)
    w["u"] = np.ones_like(w["u"])
    return orig(w, c, eps, h, st)


def _tau(w, c, eps, h, st, orig=ho.gla_step):
    return orig(w, {**c, "tau": c["tau"] * 1.25}, eps, h, st)


@pytest.mark.parametrize("kind,step", [("latent_attention", _bump_window(1)), ("latent_attention", _bump_window(-1)),
                                       ("latent_attention", _latent_with(_no_sink)), ("latent_attention", _latent_with(_base)),
                                       ("wkv", _no_shift), ("wkv", _read_first), ("gla", _tau)],
                         ids=["window+1", "window-1", "no sink", "rotation base", "no token shift", "no bonus", "tau"])
def test_planted_mistakes_show(kind, step, tmp_path, monkeypatch):
    cfg, oracle = build(tmp_path, "mixed")
    ids = prompt(cfg, 60, 3)
    want = oracle.run(ids)
    monkeypatch.setitem(ho.MIXERS, kind, step)
    oracle.reset()
    got = oracle.run(ids)
    assert rows_error(got[40:], want[40:]) > 0.05          # 500 times the 32-bit tolerance, above the bfloat16 one


def test_oracle_pieces():
    """Closed forms of the oracle's own pieces."""
    assert np.allclose(ho.gla_decay(np.array([0.0]), 2.0), 0.5 ** 0.5)
    x = np.arange(6.0)
    r = ho.rotate_pairs(x, 3, 100.0, 4)
    assert np.allclose(r[4:], x[4:]) and np.allclose(np.hypot(r[0], r[1]), np.hypot(x[0], x[1]))
    assert np.allclose(r[:2], [x[0] * np.cos(3) - x[1] * np.sin(3), x[1] * np.cos(3) + x[0] * np.sin(3)])
    p = ho.softmax_with_sink(np.array([1.0, 1.0]), 1.0)
    assert np.allclose(p, 1 / 3)
    S, o = ho.wkv_state_step(np.zeros((2, 3)), np.ones(2), np.ones(2), np.arange(3.0), np.array([2.0, 3.0]), np.zeros(2))
    assert np.allclose(o, 5 * np.arange(3.0)) and np.allclose(S, [np.arange(3.0)] * 2)
    assert isinstance(Oracle(CONFIGS["odd"], weights(CONFIGS["odd"], 2)).token(1), np.ndarray)
