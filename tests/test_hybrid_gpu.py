"""Hybrid models end to end on the GPU against the plain token-by-token oracle: prompts, portions, decoding, batches through the
serving decoder, sequences that come and go, greedy generation through the token loop and the captured decode step."""
import ctypes as C
import io
import json
import sys

import numpy as np
import pytest

from hybrid_models import CONFIGS, build, config, gla, latent, prompt, rows_error, weights, wkv
from hybrid_oracle import Oracle, write_model

pytestmark = pytest.mark.gpu

TOL = {"float32": 1e-4, "bfloat16": 4e-2}


@pytest.fixture(scope="module")
def models(libs, tmp_path_factory):
    """Folders and oracles of the test models, made once."""
    made = {}

    def get(name, seed=1):
        if (name, seed) not in made:
            folder = tmp_path_factory.mktemp(name)
            made[name, seed] = (folder, *build(folder, name, seed))
        return made[name, seed]

    yield get


def open_engine(folder, dtype, max_ctx=400, max_batch=160):
    from det_b200.engine import Engine
    return Engine.open(str(folder), dtype, max_ctx, max_batch)


def run(e, ids, cuts):
    out, at = [], 0
    for t in cuts:
        out.append(np.array(e.step(ids[at:at + t].tolist(), list(range(t)))).reshape(t, e.vocab))
        at += t
    assert at == len(ids)
    return np.concatenate(out)


CUTS = {"whole": [150], "one by one": [1] * 150, "twos and threes": [2, 3] * 30, "growing": [2, 7, 16, 33, 64, 28], "mostly decoding": [90] + [1] * 60}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_equal_the_oracle(name, dtype, models, libs):
    folder, cfg, oracle = models(name)
    ids = prompt(cfg, 150, 7)
    oracle.reset()
    want = oracle.run(ids)
    e = open_engine(folder, dtype)
    for cut in CUTS.values():
        e.reset()
        assert rows_error(run(e, ids, cut), want) < TOL[dtype], cut
    assert libs.cuda().det_last_error() == 0
    e.close()


def test_chosen_logits_and_long_steps(models):
    """Steps longer than the model's batch; wanted places in any order; none wanted."""
    folder, cfg, oracle = models("mixed")
    ids = prompt(cfg, 120, 8)
    oracle.reset()
    want = oracle.run(ids)
    e = open_engine(folder, "float32", 200, 32)
    places = [119, 0, 31, 32, 63, 5, 64]
    got = np.array(e.step(ids.tolist(), places)).reshape(-1, e.vocab)
    assert rows_error(got, want[places]) < TOL["float32"]
    e.reset()
    assert len(e.step(ids[:100].tolist(), [])) == 0
    assert rows_error(run(e, ids[100:], [1] * 20), want[100:]) < TOL["float32"]
    e.close()


def test_residual_stream_of_every_layer(models, libs):
    folder, cfg, oracle = models("mixed")
    ids = prompt(cfg, 40, 2)
    oracle.reset()
    for t in ids:
        oracle.token(t, keep_layers=True)
    want = np.array(oracle.trace).reshape(len(ids), len(cfg["layers"]), -1)
    e = open_engine(folder, "float32")
    got = {}

    def tap(user, kind, layer, pos0, t, data, n, i, rng):
        if libs.TAP_KINDS[kind] == "Residual":
            b = np.zeros((t, cfg["width"]), np.float32)
            e.h.dh_backend_read(e.backend, data, b.ctypes.data, b.size)
            got[layer] = b

    cb = libs.TAP_FN(tap)
    assert e.h.dh_model_forward_observed(e.model, ids.ctypes.data, len(ids), cb, None, 0) == 0
    for layer in range(len(cfg["layers"])):
        assert np.abs(got[layer + 1] - want[:, layer]).max() < 1e-4 * np.abs(want[:, layer]).max(), layer
    e.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sequences_come_and_go(dtype, models):
    """Interleaved sequences, ended ones giving their caches to new ones; what ran before must not show."""
    folder, cfg, oracle = models("mixed")
    e = open_engine(folder, dtype, 200, 64)
    prompts = [prompt(cfg, n, n) for n in (70, 3, 41, 1, 97)]
    want = []
    for p in prompts:
        oracle.reset()
        want.append(oracle.run(p))

    def turn(seq, p, lo, hi):
        e.swap(seq)
        out = np.array(e.step(p[lo:hi].tolist(), list(range(hi - lo)))).reshape(hi - lo, e.vocab)
        e.swap(seq)
        return out

    a, b = e.new_sequence(200), e.new_sequence(200)
    got = [turn(a, prompts[0], 0, 33)], [turn(b, prompts[1], 0, 2)]
    got[0].append(turn(a, prompts[0], 33, 70))
    got[1].append(turn(b, prompts[1], 2, 3))
    for g, w in zip(got, want):
        assert rows_error(np.concatenate(g), w) < TOL[dtype]
    for i in (2, 3, 4):
        seq = (a, b)[i % 2]
        e.clear(seq)
        cut = max(1, len(prompts[i]) // 2)
        parts = [turn(seq, prompts[i], 0, cut)] + ([turn(seq, prompts[i], cut, len(prompts[i]))] if cut < len(prompts[i]) else [])
        assert rows_error(np.concatenate(parts), want[i]) < TOL[dtype]
    e.free(a)
    e.free(b)
    e.close()


def follows(oracle, ids, out, slack):
    """Every generated token has the oracle's largest logit, to within `slack`."""
    oracle.reset()
    logits = oracle.run(ids)[-1]
    for t in out:
        assert logits.max() - logits[t] <= slack, (logits.max() - logits[t], len(out))
        logits = oracle.token(t)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation(name, models, libs):
    """Token loop, then the captured decode step from the same prompt: the same tokens, and they are the oracle's."""
    folder, cfg, oracle = models(name)
    ids = prompt(cfg, 50, 4)
    e = open_engine(folder, "float32")
    out = e.generate(ids.tolist(), 60)
    follows(oracle, ids, out, 2e-3)
    e.reset()
    assert e.h.dh_model_set_all_logits(e.model, 0) == 0
    assert e.h.dh_model_prefill(e.model, ids.ctypes.data, len(ids)) == 0
    first, rng = C.c_int32(0), C.c_uint64(0)
    assert e.h.dh_model_pick(e.model, 1, 1.0, 0, 1.0, C.byref(rng), C.byref(first)) == 0
    d = e.h.dh_graph_decoder_new(e.model)
    graph = [first.value]
    for n in (20, 39):                       # the second run replays the graph the first one captured
        buf = np.zeros(n, np.int32)
        assert e.h.dh_graph_decoder_enqueue(d, graph[-1], n, 1) == 0, e.h.dh_last_error()
        assert e.h.dh_graph_decoder_finish(d, buf.ctypes.data, n) == n
        graph += buf.tolist()
    e.h.dh_graph_decoder_free(d)
    follows(oracle, ids, graph, 2e-3)
    e.close()


def test_sampling_draws_from_the_same_stream(models):
    """Temperature, top-k and top-p go through the framework's sampler: deterministic by seed, greedy in the limit."""
    folder, cfg, _ = models("mixed")
    e = open_engine(folder, "float32")
    p = prompt(cfg, 20, 1).tolist()

    def go(**kw):
        e.reset()
        return e.generate(p, 24, **kw)

    greedy = go()
    assert go(temperature=0.9, top_k=20, top_p=0.9, seed=5) == go(temperature=0.9, top_k=20, top_p=0.9, seed=5)
    assert go(temperature=2.0, seed=5) != go(temperature=2.0, seed=6)
    assert go(temperature=1.0, top_k=1, seed=9) == greedy
    e.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n_seq", [3, 6])
def test_batched_decoder(dtype, n_seq, models, libs):
    """Unequal requests through the serving decoder (up to four rows by the GEMV, more by the batch kernels), slots used twice:
    every stream is greedy by the oracle."""
    folder, cfg, oracle = models("mixed")
    e = open_engine(folder, dtype, 160, 48)
    b = e.h.dh_batch_new(e.model, n_seq, 120)
    assert b, e.h.dh_last_error()
    slack = 5e-3 if dtype == "float32" else 0.4
    for turn in range(2):
        prompts = [prompt(cfg, n, 10 * turn + n) for n in (1, 40, 22, 77, 9, 61)[turn:turn + n_seq] + ((5,) if turn + n_seq > 6 else ())]
        for i, p in enumerate(prompts):
            assert e.h.dh_batch_prefill(b, i, p.ctypes.data, len(p), 1, 1.0, 0, 1.0, 0) == 0, e.h.dh_last_error()
        assert e.h.dh_batch_step(b, 30) == 0, e.h.dh_last_error()
        for i, p in enumerate(prompts):
            out = np.zeros(31, np.int32)
            assert e.h.dh_batch_tokens(b, i, out.ctypes.data, 31) == 31
            follows(oracle, p, out.tolist(), slack)
    e.h.dh_batch_free(b)
    assert libs.cuda().det_last_error() == 0
    e.close()


def test_batch_rows_equal_the_sequence_alone(models, libs):
    """Logits of a batched step, row by row, against the same sequence on its own."""
    folder, cfg, oracle = models("windows")
    e = open_engine(folder, "float32", 300, 64)
    lengths = [1, 17, 64, 99, 101, 130, 7]
    b = e.h.dh_batch_new(e.model, len(lengths), 200)
    prompts = [prompt(cfg, n, n) for n in lengths]
    for i, p in enumerate(prompts):
        assert e.h.dh_batch_prefill(b, i, p.ctypes.data, len(p), 1, 1.0, 0, 1.0, 0) == 0
    for _ in range(3):
        assert e.h.dh_batch_step(b, 1) == 0
    logits = np.zeros((64, e.vocab), np.float32)
    e.h.dh_model_logits(e.model, logits.ctypes.data, logits.size)
    for i, p in enumerate(prompts):
        out = np.zeros(4, np.int32)
        e.h.dh_batch_tokens(b, i, out.ctypes.data, 4)
        oracle.reset()
        want = oracle.run(np.concatenate([p, out[:3]]))[-1:]
        assert rows_error(logits[i:i + 1], want) < TOL["float32"], lengths[i]
    e.h.dh_batch_free(b)
    e.close()


def test_long_decoding(libs, tmp_path):
    """Decoding far beyond the window and the cache ring, states carried all the way."""
    cfg = config(64, 90, [latent(2, 16, 8, 16, 24, 32, 30, 48), gla(2, 16, 24, 16.0, None), wkv(2, 24, 40)])
    oracle = Oracle(cfg, write_model(tmp_path, cfg, weights(cfg, 3)))
    ids = prompt(cfg, 700, 1)
    want = oracle.run(ids)
    for dtype in TOL:
        e = open_engine(tmp_path, dtype, 700, 16)
        got = run(e, ids, [10] + [1] * 690)
        assert rows_error(got[-64:], want[-64:]) < TOL[dtype]
        assert rows_error(got, want) < TOL[dtype]
        e.close()


def test_trace_replay(models, tmp_path, monkeypatch, capsys):
    """The replay program: interleaved requests, places in any order, a slot that is given back."""
    from det_b200 import trace
    folder, cfg, oracle = models("odd")
    a, b = prompt(cfg, 30, 1), prompt(cfg, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20].tolist(), "want": [19, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:5].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[20:].tolist(), "want": [0, 9]}, {"id": "b", "tokens": b[5:].tolist(), "want": [6]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": a[:7].tolist(), "want": [6]}], "end": ["c"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert trace.main(["--model", str(folder), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "50"]) == 0
    assert [line for line in capsys.readouterr().out.split("\n") if line.startswith("done")] == [f"done {i}" for i in range(4)]
    read = lambda i: np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
    oracle.reset()
    wa = oracle.run(a)
    oracle.reset()
    wb = oracle.run(b)
    assert rows_error(read(0), wa[[19, 3]]) < TOL["float32"]
    assert not (tmp_path / "1.f32").exists()
    assert rows_error(read(2), np.array([wa[20], wa[29], wb[11]])) < TOL["float32"]
    assert rows_error(read(3), wa[6:7]) < TOL["float32"]


def test_command_line_generates(models, capsys):
    from det_b200.__main__ import main
    folder, cfg, oracle = models("mixed")
    ids = prompt(cfg, 9, 3)
    assert main(["generate", "--model", str(folder), "--dtype", "float32", "--prompt", ",".join(map(str, ids)), "--new", "7"]) == 0
    out = [int(t) for t in capsys.readouterr().out.strip().split("\n")[-1].split(",")]
    assert len(out) == 7
    follows(oracle, ids, out, 2e-3)
