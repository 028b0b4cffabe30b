"""Dopipel models end to end on the GPU against the plain token-by-token oracle: prompts, portions, decoding, sequences that come
and go, batches, greedy generation through the token loop and the captured decode step."""
import ctypes as C
import io
import json
import sys

import numpy as np
import pytest

from dopipel_models import CONFIGS, attention, build, config, dense, mingru, weights
from dopipel_oracle import Oracle
from hybrid_models import prompt, rows_error
from hybrid_oracle import write_model

pytestmark = pytest.mark.gpu

TOL = {"float32": 1e-4, "bfloat16": 5e-2}


@pytest.fixture(scope="module")
def models(libs, tmp_path_factory):
    """Folders and oracles of the test models, made once.  For bfloat16 the experts are chosen by the corrections alone: a router's
    close call could fall either way."""
    made = {}

    def get(name, dtype="float32"):
        if (name, dtype) not in made:
            folder = tmp_path_factory.mktemp(name)
            made[name, dtype] = (folder, *build(folder, name, 1, dtype == "bfloat16"))
        return made[name, dtype]

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
    folder, cfg, oracle = models(name, dtype)
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
    folder, cfg, oracle = models("mixed")
    ids = prompt(cfg, 120, 8)
    oracle.reset()
    want = oracle.run(ids)
    e = open_engine(folder, "float32", 200, 32)
    places = [119, 0, 31, 32, 63, 5, 64]
    assert rows_error(np.array(e.step(ids.tolist(), places)).reshape(-1, e.vocab), want[places]) < TOL["float32"]
    e.reset()
    assert len(e.step(ids[:100].tolist(), [])) == 0
    assert rows_error(run(e, ids[100:], [1] * 20), want[100:]) < TOL["float32"]
    e.close()


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_residual_stream_of_every_layer_run(name, models, libs):
    folder, cfg, oracle = models(name)
    ids = prompt(cfg, 40, 2)
    oracle.reset()
    for t in ids:
        oracle.token(t, keep_layers=True)
    want = np.array(oracle.trace).reshape(len(ids), len(oracle.runs), -1)
    e = open_engine(folder, "float32")
    got = {}

    def tap(user, kind, layer, pos0, t, data, n, i, rng):
        if libs.TAP_KINDS[kind] == "Residual":
            b = np.zeros((t, cfg["width"]), np.float32)
            e.h.dh_backend_read(e.backend, data, b.ctypes.data, b.size)
            got[layer] = b

    cb = libs.TAP_FN(tap)
    assert e.h.dh_model_forward_observed(e.model, ids.ctypes.data, len(ids), cb, None, 0) == 0
    assert sorted(got) == list(range(len(oracle.runs) + 1))
    for r in range(len(oracle.runs)):
        assert np.abs(got[r + 1] - want[:, r]).max() < 1e-4 * np.abs(want[:, r]).max(), r
    e.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sequences_come_and_go(dtype, models):
    """Interleaved sequences, ended ones giving their caches and states to new ones; what ran before must not show."""
    folder, cfg, oracle = models("mixed", dtype)
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
    for n in (20, 39):
        buf = np.zeros(n, np.int32)
        assert e.h.dh_graph_decoder_enqueue(d, graph[-1], n, 1) == 0, e.h.dh_last_error()
        assert e.h.dh_graph_decoder_finish(d, buf.ctypes.data, n) == n
        graph += buf.tolist()
    e.h.dh_graph_decoder_free(d)
    follows(oracle, ids, graph, 2e-3)
    e.close()


@pytest.mark.parametrize("n_seq", [3, 6])
def test_batched_decoder(n_seq, models, libs):
    """Unequal requests through the serving decoder, slots used twice: every stream is greedy by the oracle, and a row's logits are
    the sequence's own."""
    folder, cfg, oracle = models("mixed")
    e = open_engine(folder, "float32", 160, 48)
    b = e.h.dh_batch_new(e.model, n_seq, 120)
    assert b, e.h.dh_last_error()
    for turn in range(2):
        prompts = [prompt(cfg, n, 10 * turn + n) for n in (1, 40, 22, 77, 9, 61, 5)[turn:turn + n_seq]]
        for i, p in enumerate(prompts):
            assert e.h.dh_batch_prefill(b, i, p.ctypes.data, len(p), 1, 1.0, 0, 1.0, 0) == 0, e.h.dh_last_error()
        assert e.h.dh_batch_step(b, 30) == 0, e.h.dh_last_error()
        logits = np.zeros((48, e.vocab), np.float32)
        e.h.dh_model_logits(e.model, logits.ctypes.data, logits.size)
        for i, p in enumerate(prompts):
            out = np.zeros(31, np.int32)
            assert e.h.dh_batch_tokens(b, i, out.ctypes.data, 31) == 31
            follows(oracle, p, out.tolist(), 5e-3)
            oracle.reset()
            assert rows_error(logits[i:i + 1], oracle.run(np.concatenate([p, out[:30]]))[-1:]) < TOL["float32"]
    e.h.dh_batch_free(b)
    assert libs.cuda().det_last_error() == 0
    e.close()


def test_long_decoding(libs, tmp_path):
    cfg = config(64, 90, [dense(attention(4, 2, 16, 24, 12), 40), dense(mingru(48), 32)], taps=4, loop=(0, 1, 2))
    oracle = Oracle(cfg, write_model(tmp_path, cfg, weights(cfg, 3)))
    ids = prompt(cfg, 600, 1)
    want = oracle.run(ids)
    for dtype in TOL:
        e = open_engine(tmp_path, dtype, 600, 16)
        assert rows_error(run(e, ids, [10] + [1] * 590), want) < TOL[dtype]
        e.close()


def test_trace_replay(models, tmp_path, monkeypatch, capsys):
    from det_b200 import trace
    folder, cfg, oracle = models("odd")
    a, b = prompt(cfg, 30, 1), prompt(cfg, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20].tolist(), "want": [19, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[20:].tolist(), "want": [0, 9]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": b.tolist(), "want": [11]}], "end": ["b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert trace.main(["--model", str(folder), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "40"]) == 0
    assert "done 2" in capsys.readouterr().out
    oracle.reset()
    wa = oracle.run(a)
    oracle.reset()
    wb = oracle.run(b)
    read = lambda i: np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
    assert rows_error(np.concatenate([read(0), read(1), read(2)]), np.array([wa[19], wa[3], wa[20], wa[29], wb[11]])) < TOL["float32"]


def test_command_line_generates(models, capsys):
    from det_b200.__main__ import main
    folder, cfg, oracle = models("mixed")
    ids = prompt(cfg, 9, 3)
    assert main(["generate", "--model", str(folder), "--dtype", "float32", "--prompt", ",".join(map(str, ids)), "--new", "7"]) == 0
    out = [int(t) for t in capsys.readouterr().out.strip().split("\n")[-1].split(",")]
    assert len(out) == 7
    follows(oracle, ids, out, 2e-3)
