"""Inference engine of layer-list models: prompts (whole or in portions) through the tensor-core pass, decoding as one
captured token step, sequence slots with their caches and states.

:meth:`LayerEngine.step` is the serving step of one request: it runs exactly the tokens it is given, from the state earlier
steps left, and returns the logits asked for.  :meth:`prefill`, :meth:`decode_steps` and the rest of the generator's
interface run all slots together, with the same kernels.
"""
from __future__ import annotations

from typing import Hashable, Optional, Sequence

import numpy as np
import torch

from ..models.layer_list import LayerListConfig
from ..models.layer_model import LayerModel
from ..ops import _lib
from ..ops import layers as K
from ..utils import canary as CA
from .layer_cache import SlotManager
from .token_loop import TokenLoop

LOGIT_ROWS = 1024          # rows of logits computed at a time when many positions are asked for


class LayerEngine(TokenLoop):
    def __init__(self, cfg: LayerListConfig, named, batch: int = 1, max_len: int = 2048, prefill_chunk: int = 2048,
                 dtype=torch.bfloat16, device=None, gemm_min_batch: int = 8, use_tensor_cores: bool = True):
        """``batch``: sequence slots (and sequences a generation advances together).  ``max_len``: longest sequence that
        layers without a window can hold; ``prefill_chunk``: most tokens of a sequence in one pass.  From
        ``gemm_min_batch`` sequences on the token step runs its products as GEMMs."""
        self.cfg, self.B, self.cap = cfg, batch, max_len
        self.dev = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
        self.dtype = dtype
        self.chunk = max(1, min(prefill_chunk, max_len))
        # rows of one pass: the sequences of a prompt batch go through together while they fit
        rows = max(self.chunk, min(batch * self.chunk, 16384), batch)
        self.model = LayerModel(cfg, named, batch, rows, dtype, self.dev, use_tensor_cores)
        self.mem = SlotManager(cfg, batch, max_len, self.chunk, dtype, self.dev)
        self._init_loop(batch, cfg.vocab_size, max_len)
        self.weight_bytes = self.model.weight_bytes
        self.batched = batch >= gemm_min_batch if gemm_min_batch > 0 else False
        self._ids = CA.zeros(self.model.rows_max, dtype=torch.int32, device=self.dev)
        self._claimed = False

    @property
    def token_limit(self) -> Optional[int]:
        """Most tokens a sequence may have, or None."""
        return self.mem.limit

    # ------------------------------------------------------------------ one request
    def step(self, key: Hashable, tokens: Sequence[int], want: Sequence[int] = ()) -> Optional[torch.Tensor]:
        """Run the next ``tokens`` of request ``key``; fp32 logits [len(want), vocab] at the places ``want`` among them."""
        toks = np.asarray(tokens, dtype=np.int64).reshape(-1)
        want = [int(w) for w in want]
        if toks.size == 0:
            raise ValueError("a step needs at least one token")
        if toks.min() < 0 or toks.max() >= self.cfg.vocab_size:
            raise ValueError("token id outside the vocabulary")
        if any(w < 0 or w >= toks.size for w in want):
            raise ValueError("a wanted place lies outside the step")
        slot = self.mem.acquire(key)
        if self.mem.length[slot] == 0:
            self.state[slot].zero_()
        ids = torch.from_numpy(toks.astype(np.int32)).to(self.dev)
        out = torch.empty(len(want), (self.cfg.vocab_size + 7) // 8 * 8, dtype=torch.float32, device=self.dev) if want else None
        if toks.size == 1 and self.model.token_step_fits(1):
            self.mem.claim(slot, slot + 1, 1)
            self.model.forward_token(ids, self.mem, self.state, slot, 1, self.logits[slot:slot + 1])
            K.advance(self.state[slot:slot + 1], self.pos[slot:slot + 1], 1)
            for j in range(len(want)):
                out[j, :self.cfg.vocab_size] = self.logits[slot]
        else:
            for lo in range(0, toks.size, self.chunk):
                n = min(self.chunk, toks.size - lo)
                x = self._rows(ids[lo:lo + n], slot, 1, n)
                at = [(j, w - lo) for j, w in enumerate(want) if lo <= w < lo + n]
                for k in range(0, len(at), LOGIT_ROWS):
                    part = at[k:k + LOGIT_ROWS]
                    idx = torch.tensor([r for _, r in part], dtype=torch.int32, device=self.dev)
                    lg = self.model.logits_rows(x, idx, len(part), self._logit_buf())
                    out[torch.tensor([j for j, _ in part], device=self.dev), :self.cfg.vocab_size] = lg[:len(part), :self.cfg.vocab_size]
        return out[:, :self.cfg.vocab_size] if want else None

    def end(self, key: Hashable) -> None:
        """Give back what request ``key`` holds."""
        self.mem.release(key)

    def check(self, what: str = "step") -> None:
        """Raise if a kernel recorded a failure (waits for the device)."""
        _lib.check_status(self.dev, what)

    def _logit_buf(self):
        return self.model.buf("logits", (self.cfg.vocab_size + 7) // 8 * 8, torch.float32, rows=min(LOGIT_ROWS, self.model.rows_max))

    def _rows(self, ids, slot, B, n, on_layer=None):
        self.mem.claim(slot, slot + B, n)
        x = self.model.forward_rows(ids, self.mem, self.state, slot, B, n, on_layer)
        K.advance(self.state[slot:slot + B], self.pos[slot:slot + B], n)
        return x

    # ------------------------------------------------------------------ all slots together (generator interface)
    def reset(self, seed: int = 0):
        super().reset(seed)
        if self.mem.owner:
            raise RuntimeError("requests of step() are still open")
        self.mem.length = [0] * self.B

    def prefill(self, prompts: torch.Tensor):
        """``prompts``: int32 [B, n]; leaves the logits after the last prompt token in ``logits``."""
        B, n = prompts.shape
        if B != self.B or n < 1:
            raise ValueError("prefill needs [%d, n >= 1] token ids, got %s" % (self.B, tuple(prompts.shape)))
        host = prompts.cpu()
        if int(host.min()) < 0 or int(host.max()) >= self.cfg.vocab_size:
            raise ValueError("token id outside the vocabulary")
        prompts = prompts.to(self.dev, dtype=torch.int32)
        keep = min(n, self.hist_cap)
        self.history[:, :keep].copy_(prompts[:, n - keep:])
        self.hist_len.fill_(keep)
        group = max(1, min(B, self.model.rows_max // min(n, self.chunk)))
        for s0 in range(0, B, group):
            nb = min(group, B - s0)
            for lo in range(0, n, self.chunk):
                c = min(self.chunk, n - lo)
                x = self._rows(prompts[s0:s0 + nb, lo:lo + c].reshape(-1).contiguous(), s0, nb, c)
            last = torch.arange(nb, dtype=torch.int32, device=self.dev) * c + (c - 1)
            self.model.logits_rows(x, last, nb, self.logits[s0:s0 + nb])

    def _forward_token(self):
        if not self._claimed:
            self.mem.claim(0, self.B, 1)
        if self.batched or not self.model.token_step_fits(self.B):
            x = self.model.forward_rows(self.cur_tok, self.mem, self.state, 0, self.B, 1)
            self.model.logits_rows(x, None, self.B, self.logits)
        else:
            self.model.forward_token(self.cur_tok, self.mem, self.state, 0, self.B, self.logits)
        K.advance(self.state, self.pos, 1)

    def decode_steps(self, n: int, sp, use_graph: bool = True):
        self.mem.claim(0, self.B, n)
        self._claimed = True          # counted here: replays of the captured step do not pass through Python
        try:
            super().decode_steps(n, sp, use_graph)
        finally:
            self._claimed = False
