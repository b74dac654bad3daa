"""Batched serving over a prepared module with paged caches and per-sequence state (``ox_engine_*``)."""
from __future__ import annotations

import ctypes as C

import numpy as np

from . import _ffi
from ._ffi import check


class Engine:
    """`max_tokens`: tokens the live sequences may hold together, each rounded up to whole pages; `max_seqs`: live
    sequences. Sequences are fed by hand through :meth:`forward`, or submitted as requests that :meth:`step` schedules."""

    def __init__(self, session, max_tokens: int, max_seqs: int):
        self.session = session
        self._lib = _ffi.cuda_lib()
        h = C.c_void_p()
        check(self._lib.ox_engine_create(session._h, int(max_tokens), int(max_seqs), C.byref(h)))
        self._h = h
        self.vocab = self.stats()["vocab"]

    def stats(self) -> dict:
        out = (C.c_int64 * 7)()
        self._lib.ox_engine_stats(self._h, out)
        return dict(zip(("page_size", "free_pages", "free_slots", "live", "waiting", "running", "vocab"), [int(v) for v in out]))

    def forward(self, entries, logits: bool = True):
        """One batch: `entries` are (id, next tokens, places among them whose logits are wanted). Returns the wanted
        rows in entry order as f32 [wanted, vocab], or None (and does not wait) with ``logits=False``."""
        arr = (_ffi.EngineEntry * max(len(entries), 1))()
        keep, wanted = [], 0
        for i, (seq, tokens, want) in enumerate(entries):
            t = (C.c_int64 * max(len(tokens), 1))(*[int(v) for v in tokens])
            w = (C.c_int32 * max(len(want), 1))(*[int(v) for v in want])
            keep += [t, w]
            arr[i] = _ffi.EngineEntry(int(seq), t, len(tokens), w, len(want))
            wanted += len(want)
        out = np.empty((wanted, self.vocab), dtype=np.float32) if logits else None
        ptr = out.ctypes.data_as(C.POINTER(C.c_float)) if logits else None
        check(self._lib.ox_engine_forward(self._h, arr, len(entries), ptr, out.size if logits else 0))
        return out

    def release(self, seq: int) -> None:
        check(self._lib.ox_engine_release(self._h, int(seq)))

    def submit(self, prompt, max_new: int, *, eos: int = -1, temperature: float = 0.0, top_k: int = 0, top_p: float = 1.0,
               seed: int = 0) -> int:
        arr = (C.c_int64 * max(len(prompt), 1))(*[int(v) for v in prompt])
        out = C.c_int64()
        check(self._lib.ox_engine_submit(self._h, arr, len(prompt), int(max_new), int(eos), float(temperature), int(top_k), float(top_p),
                                         int(seed) & (2 ** 64 - 1), C.byref(out)))
        return out.value

    def step(self, token_budget: int = 2048) -> list:
        """One scheduler step → [(request, token, finished)]."""
        s = self.stats()
        cap = max(s["waiting"] + s["running"], 1)
        arr = (_ffi.EngineToken * cap)()
        n = C.c_int32()
        check(self._lib.ox_engine_step(self._h, int(token_budget), arr, cap, C.byref(n)))
        return [(arr[i].request, arr[i].token, bool(arr[i].finished)) for i in range(n.value)]

    def cancel(self, request: int) -> None:
        check(self._lib.ox_engine_cancel(self._h, int(request)))

    def generate(self, prompts, max_new: int, *, token_budget: int = 2048, eos: int = -1, temperature: float = 0.0,
                 top_k: int = 0, top_p: float = 1.0, seed: int = 0) -> list:
        """Generated tokens of every prompt, batched continuously."""
        ids = [self.submit(p, max_new, eos=eos, temperature=temperature, top_k=top_k, top_p=top_p, seed=seed + i)
               for i, p in enumerate(prompts)]
        out = {i: [] for i in ids}
        while True:
            s = self.stats()
            if s["waiting"] + s["running"] == 0:
                break
            for request, token, _ in self.step(token_budget):
                if request in out:
                    out[request].append(token)
        return [out[i] for i in ids]

    def close(self) -> None:
        if getattr(self, "_h", None):
            self._lib.ox_engine_free(self._h)
            self._h = None

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass
