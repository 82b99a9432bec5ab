"""What every engine on the device does around one forward pass of the next token: the sampler and its history, the random
draws, the transcript, stop tokens, and the captured decode step.

An engine provides ``_forward_token()`` (``cur_tok`` of every sequence to fp32 ``logits``, advancing the per-sequence
state) and ``prefill()``; :class:`TokenLoop` owns the buffers these meet in, so that the generator, the command line and
the benchmarks drive any of them.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence

import torch

from ..ops import decode as D
from ..utils import canary as CA


def _host():
    from .. import _gb200_host as H       # imported when something is sampled: forward passes alone do not need it
    return H


@dataclass
class SamplingParams:
    temperature: float = 0.8
    top_k: int = 40
    top_p: float = 0.92
    min_p: float = 0.05
    repetition_penalty: float = 1.12
    repetition_window: int = 128
    frequency_penalty: float = 0.0
    presence_penalty: float = 0.0
    no_repeat_ngram: int = 0
    greedy: bool = False
    seed: int = 0

    def to_native(self) -> "SamplingConfig":
        c = _host().SamplingConfig()
        for k, v in self.__dict__.items():
            setattr(c, k, v)
        c.validate()
        return c

    def device_ok(self) -> bool:
        """Settings the device sampler takes; anything else is sampled on the host from the logits."""
        if self.no_repeat_ngram > 0 or self.repetition_window > 1024:
            return False
        return self.greedy or self.temperature <= 0 or 1 <= self.top_k <= 1024


class TokenLoop:
    """Sampling state of ``B`` sequences that advance together (attributes ``B``, ``dev`` and ``cfg`` come from the engine)."""

    def _init_loop(self, B: int, V: int, max_len: int):
        f32 = dict(dtype=torch.float32, device=self.dev)
        i32 = dict(dtype=torch.int32, device=self.dev)
        self.state = CA.zeros(B, D.STATE_INTS, **i32)
        self.pos = CA.zeros(B, **i32)
        self.cur_tok = CA.zeros(B, **i32)
        self.logits = CA.zeros(B, (V + 7) // 8 * 8, **f32)[:, :V]      # rows 16-byte aligned for any vocabulary
        self.hist_cap = max_len + 8
        self.history = CA.zeros(B, self.hist_cap, **i32)
        self.hist_len = CA.zeros(B, **i32)
        self.uniforms = CA.zeros(max_len, B, **f32)      # one row of draws per sampling step
        self.tok_log = CA.zeros(B, max_len, **i32)
        self.step_no = CA.zeros(1, **i32)
        self.stop = CA.zeros(8, **i32)
        self.n_stop = 0
        self.graph: Optional[torch.cuda.CUDAGraph] = None
        self._graph_key = None
        self._rng = None
        self._uni_host = torch.zeros(max_len, B, dtype=torch.float32).pin_memory()
        self._host_step = 0

    @property
    def rng(self):
        if self._rng is None:
            self._rng = _host().Rng(1)
        return self._rng

    # ------------------------------------------------------------------ sampling
    def _sample_args(self, sp: SamplingParams) -> D.SampleArgs:
        a = D.SampleArgs()
        a.logits, a.ld, a.B, a.V = self.logits.data_ptr(), self.logits.stride(0), self.B, self.cfg.vocab_size
        n = sp.to_native()
        a.temperature, a.top_k, a.top_p, a.min_p = n.temperature, n.top_k, n.top_p, n.min_p
        a.rep_penalty, a.freq_penalty, a.presence_penalty = n.repetition_penalty, n.frequency_penalty, n.presence_penalty
        a.rep_window, a.greedy = n.repetition_window, int(n.greedy)
        a.history, a.hist_cap, a.hist_len = self.history.data_ptr(), self.hist_cap, self.hist_len.data_ptr()
        a.uniforms, a.out_tok, a.state = self.uniforms.data_ptr(), self.cur_tok.data_ptr(), self.state.data_ptr()
        a.stop, a.n_stop = self.stop.data_ptr(), self.n_stop
        a.tok_log, a.log_cap, a.step = self.tok_log.data_ptr(), self.tok_log.shape[1], self.step_no.data_ptr()
        return a

    def _step_eager(self, sp: Optional[SamplingParams]):
        self._forward_token()
        if sp is not None:
            D.sample(self._sample_args(sp))

    def decode_steps(self, n: int, sp: SamplingParams, use_graph: bool = True):
        """Run ``n`` decode steps (forward of ``cur_tok`` + sampling of the next token) without host reads."""
        if not sp.device_ok():
            raise ValueError("these sampling settings need the host sampler: use Generator.generate")
        key = (sp.temperature, sp.top_k, sp.top_p, sp.min_p, sp.repetition_penalty, sp.repetition_window,
               sp.frequency_penalty, sp.presence_penalty, sp.greedy, self.n_stop)
        self._draw_uniforms(n)
        if use_graph and (self.graph is None or self._graph_key != key):
            self._step_eager(sp)          # a real step, run eagerly: first-use set-up must happen outside capture
            n -= 1
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, capture_error_mode="thread_local"):   # other threads (prefetch, checkpoint writer) may call CUDA
                self._step_eager(sp)
            self.graph, self._graph_key = g, key
        for _ in range(max(0, n)):
            if use_graph:
                self.graph.replay()
            else:
                self._step_eager(sp)

    def _draw_uniforms(self, n: int):
        """Draws for the next ``n`` sampling steps: rows [done, done + n) of the device table the sampler indexes with
        its own step counter.  Each row is written once per generation, so the asynchronous copy never races with
        the host filling later rows."""
        lo = self._host_step
        hi = min(lo + n, self._uni_host.shape[0])
        for s in range(lo, hi):
            for b in range(self.B):
                self._uni_host[s, b] = self.rng.uniform()
        if hi > lo:
            self.uniforms[lo:hi].copy_(self._uni_host[lo:hi], non_blocking=True)
        self._host_step = lo + n

    # ------------------------------------------------------------------ a new generation
    def reset(self, seed: int = 0):
        self.state.zero_()
        self.pos.zero_()
        self.hist_len.zero_()
        self.step_no.zero_()
        self._host_step = 0
        self.rng.reseed(seed if seed else 1)

    def set_stop_tokens(self, ids: Sequence[int]):
        ids = list(ids)[:8]
        self.n_stop = len(ids)
        if ids:
            self.stop[:len(ids)].copy_(torch.tensor(ids, dtype=torch.int32))

    def sample_first(self, sp: SamplingParams):
        self._draw_uniforms(1)
        D.sample(self._sample_args(sp))

    def transcript(self, n_new: int) -> torch.Tensor:
        """Tokens sampled so far, [B, n_new] on the host (one device->host copy)."""
        return self.tok_log[:, :n_new].cpu()
