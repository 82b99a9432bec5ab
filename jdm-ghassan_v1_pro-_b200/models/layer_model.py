"""A layer-list model on the device: weights in the layout of the kernels, activation buffers, and the forward pass of new
tokens over the caches and states of ``inference/layer_cache.py``.

Two schedules of the same layers:

* :meth:`LayerModel.forward_rows`: any number of consecutive new tokens per sequence (a prompt, a portion of one, or one
  token of many sequences): tcgen05 GEMMs (fp32: the CUDA-core product), each sublayer followed by one kernel that
  normalises its output, adds it to the fp32 residual and leaves the 16-bit copy the next product reads.
* :meth:`LayerModel.forward_token`: one token of a few sequences: GEMV kernels whose prologues do those row-wise steps, so
  a layer is six (attention) or five (state-space) dependent launches, captured in one CUDA graph by the engine.

Weights are stored once.  Rows that feed a product are zero-padded to eight elements; gate and up rows are interleaved in
blocks of 64 (the layout of the fused SwiGLU epilogue); all projections that read a sublayer's input are one matrix.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from ..ops import _lib
from ..ops import gemm as G
from ..ops import layers as K
from ..utils import canary as CA
from .layer_list import AttentionMixer, LayerListConfig, Mamba2Mixer, check_tensors


SSD_MIN_TOKENS = 17       # shorter portions take the token-by-token recurrence: a chunk is 128 tokens however few are real


def _up(n: int, a: int) -> int:
    return (n + a - 1) // a * a


@dataclass
class LayerWeights:
    w_in: torch.Tensor                       # [projection rows, width]
    w_o: torch.Tensor                        # [width, mixer outputs]
    norm1: torch.Tensor
    norm2: Optional[torch.Tensor]
    w_gu: Optional[torch.Tensor]             # [2 * ff, width] interleaved
    w_down: Optional[torch.Tensor]           # [width, ff]
    vec: Dict[str, torch.Tensor]             # the mixer's small tensors, fp32


class LayerModel:
    def __init__(self, cfg: LayerListConfig, named: Dict[str, torch.Tensor], slots: int, chunk_rows: int, dtype=torch.bfloat16,
                 device=None, use_tensor_cores: bool = True):
        if dtype not in K.DTYPE:
            raise ValueError("layer-list models run in bfloat16 or float32")
        check_tensors(cfg, named)
        self.cfg, self.dtype = cfg, dtype
        self.dev = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
        self.rows_max = max(chunk_rows, slots)
        self.use_tc = use_tensor_cores and dtype == torch.bfloat16
        self.dp = _up(cfg.hidden_size, 8)
        self._load(named)
        self._bufs: Dict[tuple, torch.Tensor] = {}
        R, d = self.rows_max, cfg.hidden_size
        self.x = [CA.zeros(R, d, dtype=torch.float32, device=self.dev) for _ in range(2)]
        self.x16 = CA.zeros(R, self.dp, dtype=dtype, device=self.dev)
        self.y = CA.zeros(R, _up(d, 4), dtype=torch.float32, device=self.dev)
        self.launches = 0

    # ------------------------------------------------------------------ weights
    def _mat(self, t, cols=None, rows=None):
        """Matrix in the compute type with zero columns up to a multiple of eight."""
        r, c = t.shape
        out = CA.zeros(rows or r, _up(cols or c, 8), dtype=self.dtype, device=self.dev)
        out[:r, :c] = t.to(self.dev).to(self.dtype)
        return out

    def _vec(self, t):
        return t.to(self.dev).float().contiguous()

    def _load(self, named):
        cfg = self.cfg
        self.embed = self._mat(named["embed"])
        self.head = self._mat(named["head"])
        self.final_norm = self._vec(named["final.norm"])
        own: Dict[int, LayerWeights] = {}
        self.weights: List[LayerWeights] = []
        self.freq: List[Optional[torch.Tensor]] = []
        freq_of: Dict[object, torch.Tensor] = {}
        for spec in cfg.layers:
            j = spec.weights
            if j not in own:
                p = f"l{j}."
                m = spec.mixer
                w_in = self._mat(torch.cat([named[p + "mix." + n] for n, _ in m.projection_rows()], 0))
                stacked = {n for n, _ in m.projection_rows()} | {"o"}
                vec = {n: self._vec(named[p + "mix." + n]) for n in m.tensors(cfg.hidden_size) if n not in stacked}
                w_gu = w_down = norm2 = None
                if spec.mlp is not None:
                    E = _up(spec.mlp.ff, 64)
                    g, u = (self._mat(named[p + "mlp." + n], rows=E) for n in ("gate", "up"))
                    w_gu = G.interleave_gate_up(g.view(1, E, -1), u.view(1, E, -1)).reshape(2 * E, -1).contiguous()
                    w_down = self._mat(named[p + "mlp.down"], cols=E)
                    norm2 = self._vec(named[p + "norm2"])
                own[j] = LayerWeights(w_in, self._mat(named[p + "mix.o"]), self._vec(named[p + "norm1"]), norm2, w_gu, w_down, vec)
            self.weights.append(own[j])
            rot = getattr(spec.mixer, "rot", None)
            if rot is not None and rot.dims > 0:
                if rot not in freq_of:
                    freq_of[rot] = torch.from_numpy(rot.frequencies()).to(self.dev)
                self.freq.append(freq_of[rot])
            else:
                self.freq.append(None)
        mats = [self.head] + [t for w in own.values() for t in (w.w_in, w.w_o, w.w_gu, w.w_down) if t is not None]
        self.weight_bytes = sum(t.numel() * t.element_size() for t in mats)

    # ------------------------------------------------------------------ buffers
    def buf(self, name: str, cols: int, dtype=None, rows: int = 0) -> torch.Tensor:
        """Activation buffer shared by all layers that need one of this kind and width (padding columns stay zero)."""
        dtype = dtype or self.dtype
        key = (name, cols, dtype)
        t = self._bufs.get(key)
        if t is None:
            t = CA.zeros(rows or self.rows_max, cols, dtype=dtype, device=self.dev)
            self._bufs[key] = t
        return t

    def _scratch(self, name: str, floats: int) -> torch.Tensor:
        t = self._bufs.get((name,))
        if t is None or t.numel() < floats:
            t = torch.empty(floats, dtype=torch.float32, device=self.dev)
            self._bufs[(name,)] = t
        return t

    # ------------------------------------------------------------------ products over rows
    def _gemm(self, a, w, out, rows):
        """out[:rows] = a[:rows] @ w^T; ``out`` in the compute type or fp32."""
        self.launches += 1
        if self.dtype == torch.float32:
            K.gemm_f32(a, w, out, rows)
        else:
            G.gemm(a[:rows], w, out=out[:rows, :w.shape[0]])
        return out

    def _mlp_act(self, w: LayerWeights, rows):
        E = w.w_gu.shape[0] // 2
        act = self.buf("act", E)
        if self.dtype == torch.float32:
            gu = self.buf("gu", 2 * E)
            K.gemm_f32(self.x16, w.w_gu, gu, rows)
            K.swiglu_f32(gu, act, rows, E)
            self.launches += 2
        else:
            G.gemm_swiglu(self.x16[:rows], w.w_gu, act_out=act[:rows])
            self.launches += 1
        return act

    # ------------------------------------------------------------------ mixer arguments
    def _cs(self, freq):
        return self.buf("cs%d" % freq.data_ptr(), 2 * freq.numel(), torch.float32)

    def _rotations(self, st, B: int, n: int):
        """Cosines and sines of this pass's rows, once per distinct rotation of the model."""
        for f in {t.data_ptr(): t for t in self.freq if t is not None}.values():
            K.rotations(f, st, B, n, self._cs(f))
            self.launches += 1

    def attn_args(self, i: int, cache, st, slot: int, B: int, n: int, pos0_max: int, rotations: bool = False) -> K.AttnArgs:
        m: AttentionMixer = self.cfg.layers[i].mixer
        w = self.weights[i]
        a = K.AttnArgs()
        a.dtype, a.B, a.n, a.H, a.G = K.DTYPE[self.dtype], B, n, m.heads, m.kv_heads
        a.dk, a.dv, a.dkp, a.dvp = m.dim, m.vdim, cache.k.shape[3], cache.v.shape[3]
        f = self.freq[i]
        if f is not None:
            a.rot_dims, a.rot_half, a.freq = m.rot.dims, int(m.rot.half), f.data_ptr()
            a.cs = self._cs(f).data_ptr() if rotations else None
        a.qk_norm, a.eps, a.scale = int(m.qk_norm), self.cfg.eps, m.scale
        a.window, a.keep, a.cap = m.window, cache.keep, cache.cap
        proj = self.buf("proj", _up(w.w_in.shape[0], 8))
        a.proj, a.ld_proj, a.gate = proj.data_ptr(), proj.stride(0), int(m.gate)
        a.sink = w.vec["sink"].data_ptr() if m.sink else None
        a.q = self.buf("q", m.heads * a.dkp).data_ptr()
        a.cache_k, a.cache_v = cache.k[slot].data_ptr(), cache.v[slot].data_ptr()
        out = self.buf("mixed", w.w_o.shape[1])
        a.out, a.ldo = out.data_ptr(), out.stride(0)
        if n == 1:
            per_key_head = m.heads // m.kv_heads
            blocks = B * m.kv_heads * ((per_key_head + 3) // 4)
            seen = cache.cap if not m.window else m.window + m.keep_first
            a.splits = int(max(1, min(64, (592 + blocks - 1) // blocks, (seen + 15) // 16)))
            a.scratch = self.buf("att_scratch%d" % B, m.heads * a.splits * (a.dvp + 2), torch.float32, rows=B).data_ptr()
        a.st, a.pos0_max, a.status = st.data_ptr(), pos0_max, _lib.status_word(self.dev).data_ptr()
        return a

    def mamba_args(self, i: int, state, st, slot: int, B: int, n: int) -> K.MambaArgs:
        m: Mamba2Mixer = self.cfg.layers[i].mixer
        w = self.weights[i]
        a = K.MambaArgs()
        a.dtype, a.B, a.n = K.DTYPE[self.dtype], B, n
        a.H, a.P, a.N, a.G, a.taps = m.heads, m.vdim, m.state, m.groups, m.conv
        padx, padn = (64, 128) if self.dtype == torch.bfloat16 else (8, 8)      # whole tiles for the chunked recurrence
        a.Pp, a.Np, a.Ns = _up(m.vdim, padx), _up(m.state, padn), state.ns
        proj = self.buf("proj", _up(w.w_in.shape[0], 8))
        a.proj, a.ld_proj = proj.data_ptr(), proj.stride(0)
        v = w.vec
        a.conv_w, a.conv_b = v["conv"].data_ptr(), v["conv.b"].data_ptr()
        a.dt_bias, a.A_log, a.D = v["dt_bias"].data_ptr(), v["A_log"].data_ptr(), v["D"].data_ptr()
        a.norm_w, a.norm_groups, a.eps = v["norm"].data_ptr(), m.norm_groups, self.cfg.eps
        a.conv_state, a.ssm = state.conv[slot].data_ptr(), state.ssm[slot].data_ptr()
        tag = "%dx%d" % (m.vdim, m.state)          # padding lies inside a row: buffers are kept apart by what fills them
        a.xh = self.buf("xh" + tag, m.heads * a.Pp).data_ptr()
        a.bc, a.cc = (self.buf(s + tag, m.groups * a.Np).data_ptr() for s in ("bc", "cc"))
        y = self.buf("ssm_y", m.out_features)
        out = self.buf("mixed", w.w_o.shape[1])
        a.y, a.ld_y, a.out, a.ld_out = y.data_ptr(), y.stride(0), out.data_ptr(), out.stride(0)
        a.st, a.status = st.data_ptr(), _lib.status_word(self.dev).data_ptr()
        return a

    # ------------------------------------------------------------------ many rows
    def _mix_rows(self, i, cache, st, slot, B, n, pos0_max):
        """Mixer of layer ``i`` on the rows in ``x16``: leaves its inner output (before the output product) in "mixed"."""
        w = self.weights[i]
        self._gemm(self.x16, w.w_in, self.buf("proj", _up(w.w_in.shape[0], 8)), B * n)
        if isinstance(self.cfg.layers[i].mixer, AttentionMixer):
            a = self.attn_args(i, cache, st, slot, B, n, pos0_max, True)
            K.qkv_store(a)
            if n == 1:
                K.attn_decode(a)
            elif self.use_tc and K.attn_tc_ok(a):
                K.attn_tc(a)
            else:
                K.attn_prefill(a)
            self.launches += 2 + (n == 1)
        else:
            a = self.mamba_args(i, cache, st, slot, B, n)
            if n == 1:
                K.mamba_step(a)
            else:
                K.conv(a)
                if self.use_tc and n >= SSD_MIN_TOKENS and K.ssd_ok(a):
                    need = K.ssd_ws_floats(B, a.H, a.P, a.Ns, n)
                    if need:
                        a.chunk_ws = self._scratch("ssd", need).data_ptr()
                        self.launches += 1
                    K.ssd(a)
                else:
                    K.scan(a)
                self.launches += 1
            K.gated_norm(a)
            self.launches += 2
        return self.buf("mixed", w.w_o.shape[1])

    def forward_rows(self, ids: torch.Tensor, mem, state: torch.Tensor, slot: int, B: int, n: int, on_layer=None) -> torch.Tensor:
        """``n`` new tokens of the ``B`` sequences in slots ``slot ..`` (``ids``: int32 [B * n]); returns the residual
        [B * n, width] after the last layer.  ``state`` is advanced by the caller."""
        cfg, d, rows = self.cfg, self.cfg.hidden_size, B * n
        if rows > self.rows_max:
            raise ValueError(f"{rows} rows exceed the activation buffers ({self.rows_max})")
        st, pos0 = state[slot:], max(mem.length[slot:slot + B]) - n
        x = self.x[0]
        K.embed(ids, self.embed, x, self.x16, d)
        self.launches += 1
        self._rotations(st, B, n)
        for i, spec in enumerate(cfg.layers):
            w = self.weights[i]
            mixed = self._mix_rows(i, mem.layers[i], st, slot, B, n, pos0)
            self._gemm(mixed, w.w_o, self.y, rows)
            K.postnorm(self.y, x, w.norm1, cfg.eps, x, self.x16, rows, d)
            self.launches += 1
            if spec.mlp is not None:
                act = self._mlp_act(w, rows)
                self._gemm(act, w.w_down, self.y, rows)
                K.postnorm(self.y, x, w.norm2, cfg.eps, x, self.x16, rows, d)
                self.launches += 1
            if on_layer is not None:
                on_layer(i, x[:rows])
        return x[:rows]

    def logits_rows(self, x: torch.Tensor, row_idx: Optional[torch.Tensor], rows: int, out: torch.Tensor):
        """Final norm, output product and cap for ``rows`` rows of the residual ``x`` (those named by ``row_idx``)."""
        cfg = self.cfg
        h = self.buf("final", self.dp)
        K.norm_rows(x, row_idx, self.final_norm, cfg.eps, h, rows, cfg.hidden_size)
        self._gemm(h, self.head, out, rows)
        if cfg.logit_softcap > 0:
            K.softcap(out, rows, cfg.vocab_size, cfg.logit_softcap)
        self.launches += 2
        return out

    # ------------------------------------------------------------------ one token of a few sequences
    def token_step_fits(self, B: int) -> bool:
        item = 4 if self.dtype == torch.float32 else 2
        widest = max([self.dp] + [w.w_o.shape[1] for w in self.weights])
        return B <= K.GEMV_MAX_BATCH and B * widest * item <= K.GEMV_MAX_SMEM

    def _gemv(self, w, B, out, **kw):
        a = K.GemvArgs()
        a.W, a.fmt, a.N, a.K = w.data_ptr(), K.W_FMT[self.dtype], w.shape[0], w.shape[1]
        a.B, a.dtype, a.d = B, K.DTYPE[self.dtype], kw.pop("d")
        a.out, a.ldo, a.out_f32, a.eps = out.data_ptr(), out.stride(0), int(out.dtype == torch.float32), self.cfg.eps
        for k, v in kw.items():
            setattr(a, k, v.data_ptr() if isinstance(v, torch.Tensor) else v)
        K.gemv(a)
        self.launches += 1

    def forward_token(self, ids: torch.Tensor, mem, state: torch.Tensor, slot: int, B: int, logits: torch.Tensor):
        """The next token of ``B`` sequences in slots ``slot ..``: fp32 logits of all of them.  Nothing here depends on the
        host, so a captured graph of it can be replayed."""
        cfg, d = self.cfg, self.cfg.hidden_size
        st = state[slot:]
        x, other = self.x
        K.embed(ids, self.embed, x, self.x16, d)
        self.launches += 1
        self._rotations(st, B, 1)
        y = [self.buf("tok_y%d" % k, _up(d, 4), torch.float32, rows=K.GEMV_MAX_BATCH) for k in range(2)]
        pend = None                       # norm weight of a sublayer output in y[0] that is not yet in the residual

        def from_x(w, out, **kw):
            nonlocal x, other, pend
            if pend is None:
                self._gemv(w, B, out, prologue=1, d=d, x=x, **kw)
            else:
                self._gemv(w, B, out, prologue=1, d=d, x=x, y=y[0], ldy=y[0].stride(0), w1=pend, x_out=other, **kw)
                x, other, pend = other, x, None

        def to_y(w, norm, **kw):
            nonlocal pend
            self._gemv(w, B, y[1], **kw)
            y.reverse()
            pend = norm

        for i, spec in enumerate(cfg.layers):
            w, m, c = self.weights[i], spec.mixer, mem.layers[i]
            from_x(w.w_in, self.buf("proj", _up(w.w_in.shape[0], 8)))
            if isinstance(m, AttentionMixer):
                a = self.attn_args(i, c, st, slot, B, 1, -1, True)
                K.qkv_store(a)
                K.attn_decode(a)
                self.launches += 3
                mixed = self.buf("mixed", w.w_o.shape[1])
                to_y(w.w_o, w.norm1, prologue=0, d=m.out_features, x16=mixed, ldx=mixed.stride(0))
            else:
                a = self.mamba_args(i, c, st, slot, B, 1)
                if m.heads % m.norm_groups == 0 and m.norm_groups <= 256:
                    # the step leaves y silu(z) and sums of squares that add up to the norm's groups
                    tiles = (m.vdim + 31) // 32
                    gated = self.buf("gated", m.out_features, torch.float32, rows=K.GEMV_MAX_BATCH)
                    sq = self.buf("gated_sq", m.heads * tiles, torch.float32, rows=K.GEMV_MAX_BATCH)
                    a.gated, a.gated_sq = gated.data_ptr(), sq.data_ptr()
                    K.mamba_step(a)
                    to_y(w.w_o, w.norm1, prologue=3, d=m.out_features, v32=gated, sq=sq, n_sq=m.heads * tiles, w1=w.vec["norm"],
                         parts=m.norm_groups)
                else:
                    K.mamba_step(a)
                    to_y(w.w_o, w.norm1, prologue=2, d=m.out_features, y16=a.y, ldy16=a.ld_y, z16=a.proj, ldz=a.ld_proj,
                         w1=w.vec["norm"], parts=m.norm_groups)
                self.launches += 1
            if spec.mlp is not None:
                act = self.buf("act", w.w_gu.shape[0] // 2)
                from_x(w.w_gu, act, swiglu=1)
                to_y(w.w_down, w.norm2, prologue=0, d=w.w_down.shape[1], x16=act, ldx=act.stride(0))
        if d <= K.FINAL_NORM_MAX:
            from_x(self.head, logits, w2=self.final_norm, softcap=cfg.logit_softcap)
        else:
            K.postnorm(y[0], x, pend, cfg.eps, x, self.x16, B, d)
            h = self.buf("final", self.dp)
            K.norm_rows(x, None, self.final_norm, cfg.eps, h, B, d)
            self._gemv(self.head, B, logits, prologue=0, d=d, x16=h, ldx=h.stride(0), softcap=cfg.logit_softcap)
            self.launches += 2
