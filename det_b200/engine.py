"""A model behind the C entry points, for scripts and the command line: open any registered checkpoint (a folder with
config.json and model.safetensors, or a det GGUF), step it, generate from it, serve several sequences."""
from __future__ import annotations

import array
import ctypes as C

from . import capi

DTYPES = {"bfloat16": capi.DET_BF16, "float32": capi.DET_F32}


class EngineError(RuntimeError):
    pass


def _ids(tokens) -> tuple:
    a = array.array("i", tokens)
    return a, a.buffer_info()[0], len(a)


class Engine:
    """One loaded model on the GPU with one bound sequence; further sequences through new_sequence()."""

    def __init__(self, handle: int, backend: int):
        self.h, self.backend, self.model = capi.host(), backend, handle
        self.vocab = self.h.dh_model_vocab(handle)
        self.max_batch = self.h.dh_model_max_batch(handle)

    @classmethod
    def open(cls, path: str, dtype: str = "bfloat16", max_ctx: int = 4096, max_batch: int = 512) -> "Engine":
        h = capi.host()
        backend = h.dh_cuda_backend_new(1, 1)
        if not backend:
            raise EngineError(h.dh_last_error().decode())
        model = h.dh_model_open(backend, str(path).encode(), DTYPES[dtype], max_ctx, max_batch)
        if not model:
            err = h.dh_last_error().decode()
            h.dh_backend_free(backend)
            raise EngineError(err)
        return cls(model, backend)

    def close(self) -> None:
        if self.model:
            self.h.dh_model_free(self.model)
            self.h.dh_backend_free(self.backend)
            self.model = self.backend = None

    def _ok(self, rc: int) -> None:
        if rc != 0:
            raise EngineError(self.h.dh_last_error().decode())

    def reset(self) -> None:
        self._ok(self.h.dh_model_reset(self.model))

    def step(self, tokens, want) -> array.array:
        """Runs the tokens as the bound sequence's next ones and returns the logits at the places `want` among them, row
        after row.  Longer runs than the model's batch go through in portions."""
        out = array.array("f", bytes(4 * self.vocab * len(want)))
        slots: dict[int, list[int]] = {}
        for slot, w in enumerate(want):
            slots.setdefault(w // self.max_batch, []).append(slot)
        if any(w < 0 or w >= len(tokens) for w in want):
            raise EngineError("logits of a place outside the step asked for")
        for part, at in enumerate(range(0, len(tokens), self.max_batch)):
            keep, ids, n = _ids(tokens[at:at + self.max_batch])
            mine = slots.get(part, [])
            keep_w, rows, nw = _ids([want[s] - at for s in mine])
            self._ok(self.h.dh_model_forward_rows(self.model, ids, n, rows, nw))
            del keep, keep_w
            if not mine:
                continue
            have = self.h.dh_model_logits(self.model, None, 0)
            buf = (C.c_float * have)()
            self.h.dh_model_logits(self.model, buf, have)
            got = array.array("f", memoryview(buf).cast("B").cast("f")[:nw * self.vocab])
            for i, s in enumerate(mine):
                out[s * self.vocab:(s + 1) * self.vocab] = got[i * self.vocab:(i + 1) * self.vocab]
        return out

    def generate(self, prompt, n_new: int, temperature: float = 0.0, top_k: int = 0, top_p: float = 1.0, seed: int = 0) -> list[int]:
        """Continues the bound sequence by the prompt and n_new tokens; temperature 0 is greedy."""
        keep, ids, n = _ids(prompt)
        out, n_out = (C.c_int32 * max(1, n_new))(), C.c_size_t(0)
        greedy = temperature <= 0.0
        self._ok(self.h.dh_model_generate(self.model, ids, n, n_new, int(greedy), 1.0 if greedy else 1.0 / temperature, top_k,
                                          top_p, seed, out, C.byref(n_out)))
        del keep
        return list(out[:n_out.value])

    # ---- further sequences
    def new_sequence(self, ctx: int) -> int:
        s = self.h.dh_seq_new(self.model, ctx)
        if not s:
            raise EngineError(self.h.dh_last_error().decode())
        return s

    def swap(self, seq: int) -> None:
        self._ok(self.h.dh_seq_swap(self.model, seq))

    def clear(self, seq: int) -> None:
        self._ok(self.h.dh_seq_clear(self.model, seq))

    def free(self, seq: int) -> None:
        self.h.dh_seq_free(seq)
