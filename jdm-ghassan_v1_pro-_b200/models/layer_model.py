"""A layer-list model on the device: weights in the layout of the kernels, activation buffers, and the forward pass of new
tokens over the caches and states of ``inference/layer_cache.py``.

Two schedules of the same layers:

* :meth:`LayerModel.forward_rows`: any number of consecutive new tokens per sequence (a prompt, a portion of one, or one
  token of many sequences): tcgen05 GEMMs (fp32: the CUDA-core product), each sublayer followed by one kernel that
  normalises its output, adds it to the fp32 residual and leaves the 16-bit copy the next product reads (where sublayers
  stand side by side: adds their sum to the residual and leaves the norm of that).
* :meth:`LayerModel.forward_token`: one token of a few sequences: GEMV kernels whose prologues do those row-wise steps, so
  a layer is six (attention) or five (state-space) dependent launches, captured in one CUDA graph by the engine.  Side by
  side: five (attention) or six (latent attention).

Weights are stored once.  Rows that feed a product are zero-padded to eight elements; gate and up rows are interleaved in
blocks of 64 (the layout of the fused SwiGLU epilogue); all projections that read a sublayer's input are one matrix.  Where
sublayers stand side by side, that matrix has the feed-forward's rows, too, and the two output products are one over the
concatenation of the sublayers' inner outputs.  A latent's key and value maps are one matrix in the padded layout of the
attention kernels, whose rows also carry the shared key part into every head's key.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from ..ops import _lib
from ..ops import gemm as G
from ..ops import layers as K
from ..utils import canary as CA
from .layer_list import AttentionMixer, LatentAttentionMixer, LayerListConfig, Mamba2Mixer, check_tensors


LATENT_FEW = 4            # portions up to this long attend to the latents themselves instead of keys and values made from them
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
    norm1_b: Optional[torch.Tensor] = None
    # sublayers side by side: w_in's rows are followed by the feed-forward's (w_up) in w_all, and w_o holds the mixer's
    # output columns, then (from column `off`) the feed-forward's
    w_all: Optional[torch.Tensor] = None
    w_up: Optional[torch.Tensor] = None
    off: int = 0
    w_uq: Optional[torch.Tensor] = None      # latent attention: queries from their latent
    w_kv: Optional[torch.Tensor] = None      # [H * dkp + H * dvp, latent row] keys and values from cache rows


class LayerModel:
    def __init__(self, cfg: LayerListConfig, named: Dict[str, torch.Tensor], slots: int, chunk_rows: int, dtype=torch.bfloat16,
                 device=None, use_tensor_cores: bool = True):
        if dtype not in K.DTYPE:
            raise ValueError("layer-list models run in bfloat16 or float32")
        check_tensors(cfg, named)
        self.cfg, self.dtype = cfg, dtype
        self.dev = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
        self.rows_max = max(chunk_rows, slots)
        self.parallel = cfg.design.block == "parallel"
        self.use_tc = use_tensor_cores and dtype == torch.bfloat16
        self.dp = _up(cfg.hidden_size, 8)
        self._load(named)
        self._bufs: Dict[tuple, torch.Tensor] = {}
        R, d = self.rows_max, cfg.hidden_size
        self.x = [CA.zeros(R, d, dtype=torch.float32, device=self.dev) for _ in range(2)]
        self.x0 = CA.zeros(R, d, dtype=torch.float32, device=self.dev) if self.parallel else None      # embedding output
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

    def _norm(self, named, name):
        """(weight, bias or None) of a norm."""
        return self._vec(named[name]), self._vec(named[name + ".b"]) if self.cfg.design.norm == "layer" else None

    def _load(self, named):
        cfg = self.cfg
        self.embed = self._mat(named["embed"])
        self.head = self._mat(named["head"])
        self.embed_norm = self._norm(named, "embed.norm") if cfg.design.embed_norm else None
        self.final_norm, self.final_norm_b = self._norm(named, "final.norm")
        own: Dict[int, LayerWeights] = {}
        self.weights: List[LayerWeights] = []
        self.freq: List[Optional[torch.Tensor]] = []
        self.slopes: List[Optional[torch.Tensor]] = []
        freq_of: Dict[object, torch.Tensor] = {}
        for spec in cfg.layers:
            j = spec.weights
            if j not in own:
                own[j] = (self._load_parallel if self.parallel else self._load_post)(named, j, spec)
            self.weights.append(own[j])
            m = spec.mixer
            rot = getattr(m, "rot", None)
            if rot is not None and rot.dims > 0:
                if rot not in freq_of:
                    freq_of[rot] = torch.from_numpy(rot.frequencies()).to(self.dev)
                self.freq.append(freq_of[rot])
            else:
                self.freq.append(None)
            self.slopes.append(torch.from_numpy(m.slopes()).float().to(self.dev) if getattr(m, "distance_bias", False) else None)
        mats = [self.head] + [t for w in own.values() for t in (w.w_in if w.w_all is None else w.w_all, w.w_o, w.w_gu, w.w_down, w.w_uq, w.w_kv)
                              if t is not None]
        self.weight_bytes = sum(t.numel() * t.element_size() for t in mats)

    def _mixer_vec(self, named, p, m):
        """The mixer's tensors that no product reads."""
        mats = {n for n, _ in m.projection_rows()} | {"o"} | ({"uq", "uk", "uv"} if isinstance(m, LatentAttentionMixer) else set())
        return {n: self._vec(named[p + "mix." + n]) for n in m.tensors(self.cfg.hidden_size) if n not in mats}

    def _load_post(self, named, j, spec) -> LayerWeights:
        p, m = f"l{j}.", spec.mixer
        w_in = self._mat(torch.cat([named[p + "mix." + n] for n, _ in m.projection_rows()], 0))
        w_gu = w_down = norm2 = None
        if spec.mlp is not None:
            E = _up(spec.mlp.ff, 64)
            g, u = (self._mat(named[p + "mlp." + n], rows=E) for n in ("gate", "up"))
            w_gu = G.interleave_gate_up(g.view(1, E, -1), u.view(1, E, -1)).reshape(2 * E, -1).contiguous()
            w_down = self._mat(named[p + "mlp.down"], cols=E)
            norm2 = self._vec(named[p + "norm2"])
        return LayerWeights(w_in, self._mat(named[p + "mix.o"]), self._vec(named[p + "norm1"]), norm2, w_gu, w_down, self._mixer_vec(named, p, m))

    def _load_parallel(self, named, j, spec) -> LayerWeights:
        p, m = f"l{j}.", spec.mixer
        rows = [named[p + "mix." + n] for n, _ in m.projection_rows()]
        n_in = sum(t.shape[0] for t in rows)
        w_o, off, w_up = named[p + "mix.o"], 0, None
        if spec.mlp is not None:
            off = _up(m.out_features, 8)
            w_o = torch.cat([w_o, w_o.new_zeros(w_o.shape[0], off - m.out_features), named[p + "mlp.down"]], 1)
            rows.append(named[p + "mlp.up"])
        w_all = self._mat(torch.cat(rows, 0))
        if spec.mlp is not None:
            w_up = w_all[n_in:]
        norm1, norm1_b = self._norm(named, p + "norm1")
        w = LayerWeights(w_all[:n_in], self._mat(w_o), norm1, None, None, None, self._mixer_vec(named, p, m), norm1_b, w_all, w_up, off)
        if isinstance(m, LatentAttentionMixer):
            H, R = m.heads, m.kv_rank
            dkp, dvp, ldc = K.head_pad(m.dim + m.rot_dim, self.dtype), K.head_pad(m.vdim, self.dtype), _up(R + m.rot_dim, 8)
            w.w_uq = self._mat(named[p + "mix.uq"])
            w.w_kv = CA.zeros(H * (dkp + dvp), ldc, dtype=self.dtype, device=self.dev)
            keys, values = w.w_kv[:H * dkp].view(H, dkp, ldc), w.w_kv[H * dkp:].view(H, dvp, ldc)
            keys[:, :m.dim, :R] = named[p + "mix.uk"].to(self.dev).to(self.dtype).view(H, m.dim, R)
            keys[:, m.dim:m.dim + m.rot_dim, R:R + m.rot_dim] = torch.eye(m.rot_dim, dtype=self.dtype, device=self.dev)
            values[:, :m.vdim, :R] = named[p + "mix.uv"].to(self.dev).to(self.dtype).view(H, m.vdim, R)
        return w

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

    def mixed(self, i: int) -> torch.Tensor:
        """What the output product of layer ``i`` reads: the mixer's inner output, behind it (side by side) the feed-forward's."""
        w, spec = self.weights[i], self.cfg.layers[i]
        return self.buf("mixed" if not w.off else "mixed%d+%d" % (spec.mixer.out_features, spec.mlp.ff), w.w_o.shape[1])

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
        a.proj, a.ld_proj = proj.data_ptr(), proj.stride(0)
        if m.gate:
            a.gate, a.ld_gate = proj[:, (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim:].data_ptr(), proj.stride(0)
        a.sink = w.vec["sink"].data_ptr() if m.sink else None
        a.softcap, a.slopes = m.softcap, None if self.slopes[i] is None else self.slopes[i].data_ptr()
        if m.q_temp is not None:
            a.temp_coef, a.temp_every = m.q_temp.coef, m.q_temp.every
        a.q = self.buf("q", m.heads * a.dkp).data_ptr()
        a.cache_k, a.cache_v, a.ld_k, a.ld_v = cache.k[slot].data_ptr(), cache.v[slot].data_ptr(), m.kv_heads * a.dkp, m.kv_heads * a.dvp
        out = self.mixed(i)
        a.out, a.ldo = out.data_ptr(), out.stride(0)
        if n == 1:
            per_key_head = m.heads // m.kv_heads
            blocks = B * m.kv_heads * ((per_key_head + 3) // 4)
            seen = cache.cap if not m.window else m.window + m.keep_first
            a.splits = int(max(1, min(64, (592 + blocks - 1) // blocks, (seen + 15) // 16)))
            a.scratch = self.buf("att_scratch%d" % B, m.heads * a.splits * (a.dvp + 2), torch.float32, rows=B).data_ptr()
        a.st, a.pos0_max, a.status = st.data_ptr(), pos0_max, _lib.status_word(self.dev).data_ptr()
        return a

    def latent_args(self, i: int, cache, st, slot: int, B: int, n: int) -> K.LatentArgs:
        m: LatentAttentionMixer = self.cfg.layers[i].mixer
        w, rows = self.weights[i], B * n
        a = K.LatentArgs()
        a.dtype, a.B, a.n = K.DTYPE[self.dtype], B, n
        a.H, a.dn, a.dr, a.dv, a.rank, a.q_rank = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.q_rank
        a.dkp, a.dvp = K.head_pad(m.dim + m.rot_dim, self.dtype), K.head_pad(m.vdim, self.dtype)
        if self.freq[i] is not None:
            a.rot_dims, a.cs = m.rot.dims, self._cs(self.freq[i]).data_ptr()
        a.eps, a.scale = self.cfg.eps, m.scale
        proj, cq = self.buf("proj", _up(w.w_in.shape[0], 8)), self.buf("cq", w.w_uq.shape[1])
        a.proj, a.ld_proj, a.q_norm, a.kv_norm = proj.data_ptr(), proj.stride(0), w.vec["dq.norm"].data_ptr(), w.vec["dkv.norm"].data_ptr()
        a.cq, a.ld_cq = cq.data_ptr(), cq.stride(0)
        a.cache, a.ldc, a.cap = cache.rows[slot].data_ptr(), cache.rows.shape[2], cache.cap
        qc = self.buf("qc", _up(w.w_uq.shape[0], 8))
        a.qc, a.ld_qc, a.W_kv, a.ld_w = qc.data_ptr(), qc.stride(0), w.w_kv.data_ptr(), w.w_kv.stride(0)
        a.gate, a.ld_gate = proj[:, m.q_rank + m.kv_rank + m.rot_dim:].data_ptr(), proj.stride(0)
        out = self.mixed(i)
        a.out, a.ldo = out.data_ptr(), out.stride(0)
        if n <= LATENT_FEW:
            plan = K.latent_tc_plan(a) if self.use_tc else None
            if plan is not None:
                a.heads_pad, a.ld_qa16 = plan
                a.qa16 = self.buf("qa16:%dx%d+%d" % (rows, m.heads, m.kv_rank + m.rot_dim), a.heads_pad * a.ld_qa16, rows=rows).data_ptr()
                a.splits = int(max(1, min(64, 148 // (rows * ((m.heads + 31) // 32)), cache.cap // 128)))
            else:
                a.qa = self.buf("qa%d" % rows, m.heads * a.ldc, torch.float32, rows=rows).data_ptr()
                blocks = rows * ((m.heads + 3) // 4)
                a.splits = int(max(1, min(64, (592 + blocks - 1) // blocks, (cache.cap + 15) // 16)))
            a.scratch = self.buf("latent_scratch%d" % rows, m.heads * a.splits * (a.ldc + 2), torch.float32, rows=rows).data_ptr()
        else:
            a.q = self.buf("q", m.heads * a.dkp).data_ptr()
        a.st, a.status = st.data_ptr(), _lib.status_word(self.dev).data_ptr()
        return a

    def _expanded(self, i: int, cache, slot: int, B: int, ctx: int):
        """Keys and values of the first ``ctx`` positions of ``B`` sequences, made from their latents: ([rows, H * dkp + H * dvp],
        rows per sequence).  Rows up to the next whole key tile are finite, whatever they hold."""
        w, rows = self.weights[i].w_kv, cache.rows[slot:slot + B]
        per = min(_up(ctx, 128), cache.cap)
        if B > 1 and cache.cap <= 2 * per:                  # one product over the slots as they lie
            per = cache.cap
        need, cols = B * per, w.shape[0]
        kv = self._bufs.get(("kv", cols))
        if kv is None or kv.shape[0] < need:
            kv = torch.zeros(need, cols, dtype=self.dtype, device=self.dev)
            self._bufs[("kv", cols)] = kv
        if per == cache.cap:
            self._gemm(rows.view(B * per, -1), w, kv, need)
        else:
            for b in range(B):
                self._gemm(rows[b], w, kv[b * per:], per)
        return kv, per

    def expanded_attn_args(self, i: int, a: K.LatentArgs, kv: torch.Tensor, per: int, pos0_max: int) -> K.AttnArgs:
        """Arguments of the attention kernels on keys and values made by :meth:`_expanded`."""
        t = K.AttnArgs()
        t.dtype, t.B, t.n, t.H, t.G = a.dtype, a.B, a.n, a.H, a.H
        t.dk, t.dv, t.dkp, t.dvp, t.eps, t.scale, t.cap = a.dn + a.dr, a.dv, a.dkp, a.dvp, a.eps, a.scale, per
        t.gate, t.ld_gate, t.q = a.gate, a.ld_gate, a.q
        t.cache_k, t.cache_v, t.ld_k, t.ld_v = kv.data_ptr(), kv[:, a.H * a.dkp:].data_ptr(), kv.stride(0), kv.stride(0)
        t.out, t.ldo, t.st, t.pos0_max, t.status = a.out, a.ldo, a.st, pos0_max, a.status
        return t

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
        out = self.mixed(i)
        a.y, a.ld_y, a.out, a.ld_out = y.data_ptr(), y.stride(0), out.data_ptr(), out.stride(0)
        a.st, a.status = st.data_ptr(), _lib.status_word(self.dev).data_ptr()
        return a

    # ------------------------------------------------------------------ many rows
    def _mix_rows(self, i, cache, st, slot, B, n, pos0_max):
        """Mixer of layer ``i`` on the rows in ``x16``: leaves its inner output (before the output product) in "mixed"."""
        w, m = self.weights[i], self.cfg.layers[i].mixer
        self._gemm(self.x16, w.w_in, self.buf("proj", _up(w.w_in.shape[0], 8)), B * n)
        if isinstance(m, AttentionMixer):
            a = self.attn_args(i, cache, st, slot, B, n, pos0_max, True)
            K.qkv_store(a)
            if n == 1:
                K.attn_decode(a)
            else:
                self._attn(a)
            self.launches += 2 + (n == 1)
        elif isinstance(m, LatentAttentionMixer):
            a = self.latent_args(i, cache, st, slot, B, n)
            K.latent_store(a)
            self._gemm(self.buf("cq", w.w_uq.shape[1]), w.w_uq, self.buf("qc", _up(w.w_uq.shape[0], 8)), B * n)
            if n <= LATENT_FEW:
                K.latent_absorb(a, False)
                K.latent_attn(a)
                self.launches += 4
            else:
                K.latent_queries(a)
                kv, per = self._expanded(i, cache, slot, B, pos0_max + n)
                self._attn(self.expanded_attn_args(i, a, kv, per, pos0_max))
                self.launches += 3
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
        return self.mixed(i)

    def _attn(self, a):
        if self.use_tc and K.attn_tc_ok(a):
            K.attn_tc(a)
        else:
            K.attn_prefill(a)

    def forward_rows(self, ids: torch.Tensor, mem, state: torch.Tensor, slot: int, B: int, n: int, on_layer=None) -> torch.Tensor:
        """``n`` new tokens of the ``B`` sequences in slots ``slot ..`` (``ids``: int32 [B * n]); returns the residual
        [B * n, width] after the last layer.  ``state`` is advanced by the caller."""
        rows = B * n
        if rows > self.rows_max:
            raise ValueError(f"{rows} rows exceed the activation buffers ({self.rows_max})")
        st, pos0 = state[slot:], max(mem.length[slot:slot + B]) - n
        return (self._rows_parallel if self.parallel else self._rows_post)(ids, mem, st, slot, B, n, pos0, on_layer)

    def _rows_post(self, ids, mem, st, slot, B, n, pos0, on_layer):
        cfg, d, rows, x = self.cfg, self.cfg.hidden_size, B * n, self.x[0]
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

    def _embed_first(self, ids, rows):
        """Embedding output into ``x0``."""
        if self.embed_norm is None:
            K.embed(ids, self.embed, self.x0, self.x16, self.cfg.hidden_size)
        else:
            K.embed_norm(ids, self.embed, (self.cfg.design.norm,) + self.embed_norm, self.cfg.eps, self.x0[:rows], self.dtype)
        self.launches += 1

    def _up_rows(self, i, rows):
        """Feed-forward rows of the input product, squared where positive, behind the mixer's columns of "mixed"."""
        w = self.weights[i]
        act = self.mixed(i)[:, w.off:]
        if self.dtype == torch.float32:
            K.gemm_f32(self.x16, w.w_up, act, rows)
            K.relu2_f32(act, rows, w.w_up.shape[0])
            self.launches += 2
        else:
            G.gemm(self.x16[:rows], w.w_up, out=act[:rows, :w.w_up.shape[0]], relu2=True)
            self.launches += 1

    def _rows_parallel(self, ids, mem, st, slot, B, n, pos0, on_layer):
        cfg, rows, x, y = self.cfg, B * n, self.x0, None
        norm = lambda w: (cfg.design.norm, w.norm1, w.norm1_b)
        self._embed_first(ids, rows)
        self._rotations(st, B, n)
        for r, run in enumerate(cfg.runs):
            i, w, first = run.layer, self.weights[run.layer], self.x0 if run.rejoin else None
            new = None if y is None and first is None else self.x[0]
            K.add_norm(x, rows, norm(w), cfg.eps, self.x16, y, cfg.residual_mult, first, new)
            x = x if new is None else new
            self._mix_rows(i, mem.layers[r], st, slot, B, n, pos0)
            if w.w_up is not None:
                self._up_rows(i, rows)
            self._gemm(self.mixed(i), w.w_o, self.y, rows)
            y = self.y[:, :cfg.hidden_size]
            self.launches += 1
            if on_layer is not None or r == len(cfg.runs) - 1:
                K.add_norm(x, rows, y=y, alpha=cfg.residual_mult, x_out=self.x[0])
                x, y = self.x[0], None
                self.launches += 1
            if on_layer is not None:
                on_layer(r, x[:rows])
        return x[:rows]

    def logits_rows(self, x: torch.Tensor, row_idx: Optional[torch.Tensor], rows: int, out: torch.Tensor):
        """Final norm, output product and cap for ``rows`` rows of the residual ``x`` (those named by ``row_idx``)."""
        cfg = self.cfg
        h = self.buf("final", self.dp)
        if cfg.design.norm == "rms":
            K.norm_rows(x, row_idx, self.final_norm, cfg.eps, h, rows, cfg.hidden_size)
        else:
            K.add_norm(x, rows, (cfg.design.norm, self.final_norm, self.final_norm_b), cfg.eps, h, row_idx=row_idx)
        self._gemm(h, self.head, out, rows)
        if cfg.logit_softcap > 0:
            K.softcap(out, rows, cfg.vocab_size, cfg.logit_softcap)
        self.launches += 2
        return out

    # ------------------------------------------------------------------ one token of a few sequences
    def token_step_fits(self, B: int) -> bool:
        item = 4 if self.dtype == torch.float32 else 2
        if self.parallel:
            widest = max([self.dp] + [w.w_uq.shape[1] for w in self.weights if w.w_uq is not None])
        else:
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
        if self.parallel:
            return self._token_parallel(ids, mem, state[slot:], slot, B, logits)
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
                mixed = self.mixed(i)
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

    def _token_parallel(self, ids, mem, st, slot, B, logits):
        cfg, d = self.cfg, self.cfg.hidden_size
        mode = K.NORM[cfg.design.norm]
        x, other, y = self.x0, self.x, None
        self._embed_first(ids, B)
        self._rotations(st, B, 1)

        def from_x(w, out, weight, bias, first=None, **kw):
            """Product of the normed residual, after what is still to be added to it."""
            nonlocal x, y
            kw.update(prologue=5, d=d, x=x, w1=weight, norm_mode=mode)
            if bias is not None:
                kw["b1"] = bias
            if first is not None:
                kw["x0"] = first
            if y is not None:
                kw.update(y=y, ldy=y.stride(0), alpha=cfg.residual_mult)
            if y is not None or first is not None:
                new = other[0] if x is not other[0] else other[1]
                self._gemv(w, B, out, x_out=new, **kw)
                x, y = new, None
            else:
                self._gemv(w, B, out, **kw)

        for r, run in enumerate(cfg.runs):
            i, m, w, c = run.layer, cfg.layers[run.layer].mixer, self.weights[run.layer], mem.layers[r]
            mixed, proj = self.mixed(i), self.buf("proj", _up(w.w_in.shape[0], 8))
            split = {} if w.w_up is None else dict(n1=w.w_in.shape[0], out2=mixed[:, w.off:], ldo2=mixed.stride(0))
            from_x(w.w_all, proj, w.norm1, w.norm1_b, self.x0 if run.rejoin else None, **split)
            if isinstance(m, AttentionMixer):
                a = self.attn_args(i, c, st, slot, B, 1, -1, True)
                K.qkv_store(a)
                K.attn_decode(a)
            else:
                a = self.latent_args(i, c, st, slot, B, 1)
                self._gemv(w.w_uq, B, self.buf("qc", _up(w.w_uq.shape[0], 8)), prologue=4, d=m.q_rank, x16=proj, ldx=proj.stride(0), w1=w.vec["dq.norm"])
                K.latent_absorb(a, True)
                K.latent_attn(a)
            self.launches += 3
            y = self.buf("tok_y0", _up(d, 4), torch.float32, rows=K.GEMV_MAX_BATCH)
            self._gemv(w.w_o, B, y, prologue=0, d=w.w_o.shape[1], x16=mixed, ldx=mixed.stride(0))
        from_x(self.head, logits, self.final_norm, self.final_norm_b)
