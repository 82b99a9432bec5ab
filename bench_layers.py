#!/usr/bin/env python
"""Layer-list models at the sizes of real models' layers, beside this framework's closest other model at equal size.

    python bench.py --layer-list [--design zikedra|dunavik] [--sizes s,m,l] [--prompt 8192] [--new 128] [--only kernels|models]

(``bench.py --layer-list`` ends up here.)  Random weights, random token ids, one B200.  Two parts:

* ``models``: prompt and decode throughput of a model of attention and Mamba-2 layers (one attention layer in four), or
  (``--design dunavik``) of window attention and latent attention (one latent layer in four) with side-by-side sublayers, and
  of the dense decoder with the same width, depth, heads, window and feed-forward (``models/config.py``, fp16).
* ``kernels``: device time of every kernel of both models on one layer's shapes, the bytes or operations the step needs,
  and the fraction of the measured copy bandwidth or tensor throughput (``MEASURED_PEAKS.json``) that this is.

Prompt kernels are timed with CUDA events, one launch per pair, with an L2-sized buffer written between them.  Kernels of
the token step are timed as a captured chain of launches over enough copies of their operands to exceed L2.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import sys

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

SIZES = {   # width, ff, query heads, kv heads, head size, mamba heads, groups, layers
    "s": dict(width=1024, ff=2816, H=16, G=4, hd=64, mh=32, mg=1, layers=12),
    "m": dict(width=2560, ff=6912, H=20, G=5, hd=128, mh=80, mg=1, layers=12),
    "l": dict(width=4096, ff=14336, H=32, G=8, hd=128, mh=128, mg=8, layers=8),
}
LATENT = {  # latent attention: unrotated / rotated / value head size, latent sizes
    "s": dict(dim=64, rot_dim=32, vdim=64, kv_rank=256, q_rank=512),
    "m": dict(dim=64, rot_dim=64, vdim=128, kv_rank=512, q_rank=768),
    "l": dict(dim=64, rot_dim=64, vdim=128, kv_rank=512, q_rank=1536),
}
WINDOW, KEEP, VOCAB, STATE, VDIM = 1024, 8, 32000, 128, 64


def peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        with open(p) as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def layer_config(z, layers=None):
    from ghassan_b200.models.layer_list import LayerListConfig
    mlp = {"kind": "dense", "ff": z["ff"]}
    at = {"type": "attention", "mlp": mlp,
          "mixer": {"heads": z["H"], "kv_heads": z["G"], "dim": z["hd"], "vdim": z["hd"], "scale": z["hd"] ** -0.5,
                    "mask": {"size": WINDOW, "keep_first": KEEP}, "rot": {"base": 500000.0, "dims": z["hd"], "scaling": None}}}
    mb = {"type": "mamba2", "mlp": mlp, "mixer": {"heads": z["mh"], "vdim": VDIM, "state": STATE, "groups": z["mg"], "conv": 4,
                                                  "norm_groups": z["mg"]}}
    n = layers or z["layers"]
    return LayerListConfig.from_json({"architecture": "Zikedra", "layers": [at if i % 4 == 3 else mb for i in range(n)], "width": z["width"],
                                      "vocab": VOCAB, "norm": {"eps": 1e-5}, "logit_softcap": 30.0})


def side_config(name, layers=None):
    """Window attention with every fourth layer a latent one; the model of :func:`dense_config` with side-by-side sublayers."""
    from ghassan_b200.models.layer_list import LayerListConfig
    z, la = SIZES[name], LATENT[name]
    mlp = {"kind": "dense", "ff": z["ff"]}
    at = {"type": "attention", "mlp": mlp,
          "mixer": {"heads": z["H"], "kv_heads": z["G"], "dim": z["hd"], "vdim": z["hd"], "scale": z["hd"] ** -0.5, "softcap": 30.0,
                    "mask": {"size": WINDOW}, "q_temp": {"coef": 0.1, "every": 4096}}}
    lt = {"type": "latent_attention", "mlp": mlp,
          "mixer": dict(la, heads=z["H"], scale=(la["dim"] + la["rot_dim"]) ** -0.5, rot={"base": 500000.0, "dims": la["rot_dim"]})}
    n = layers or z["layers"]
    return LayerListConfig.from_json({"architecture": "Dunavik", "layers": [lt if i % 4 == 3 else at for i in range(n)], "width": z["width"],
                                      "vocab": VOCAB, "norm": {"eps": 1e-5}, "residual_mult": 0.5})


def dense_config(z, layers=None):
    from ghassan_b200.models.config import ModelConfig
    return ModelConfig(vocab_size=VOCAB, hidden_size=z["width"], num_layers=layers or z["layers"], num_heads=z["H"], num_kv_heads=z["G"],
                       intermediate_size=z["ff"], max_seq_len=16384, use_moe=False, use_qk_norm=True, sliding_window=WINDOW)


def random_named(cfg):
    """fp32 host arrays of the dense model, drawn on the device."""
    import torch
    out = {}
    for s in cfg.param_specs():
        out[s.name] = (torch.ones(s.shape) if s.init == "ones" else (torch.randn(s.shape, device="cuda") * 0.02).cpu()).numpy()
    return out


class Flush:
    def __init__(self):
        import torch
        self.buf = torch.zeros(256 << 20, dtype=torch.uint8, device="cuda")

    def __call__(self):
        self.buf.zero_()


def time_launch(fn, flush, iters=15):
    """Median microseconds of one call, with L2 flushed before each."""
    import torch
    for _ in range(3):
        fn()
    torch.cuda.synchronize()
    out = []
    for _ in range(iters):
        flush()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        out.append(a.elapsed_time(b) * 1e3)
    return statistics.median(out)


def time_chain(fns, iters=10):
    """Mean microseconds per call of a captured chain of calls (each on its own copy of the operands)."""
    import torch
    for f in fns[:2]:
        f()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for f in fns:
            f()
    for _ in range(3):
        g.replay()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(iters):
        g.replay()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) * 1e3 / (iters * len(fns))


class Table:
    """Rows of the kernel table: achieved time against the time that bytes or operations alone would take."""

    def __init__(self, size, prompt):
        self.size, self.prompt = size, prompt
        self.hbm, self.tf, self.src = peaks()

    def add(self, model, kernel, us, nbytes=0.0, flops=0.0, like=""):
        need = max(nbytes / self.hbm, flops / self.tf) * 1e6
        print(json.dumps({"size": self.size, "model": model, "kernel": kernel, "like": like, "us": round(us, 2),
                          "bound": "bytes" if nbytes / self.hbm >= flops / self.tf else "flops", "of_roofline": round(need / us, 3),
                          "prompt": self.prompt, "peaks": self.src}), flush=True)


def copies(nbytes):
    """Operand copies whose sum exceeds L2 well."""
    return max(8, min(64, int(300e6 // max(1, nbytes)) + 1))


def prompt_kernels(t, z, m, mem, st, ids, T):
    import torch
    from ghassan_b200.ops import gemm as G
    from ghassan_b200.ops import kernels as KK
    from ghassan_b200.ops import layers as K
    flush = Flush()
    d, E, H, Gq, hd = z["width"], z["ff"], z["H"], z["G"], z["hd"]
    f16 = dict(dtype=torch.float16, device="cuda")
    run = lambda fn: time_launch(fn, flush)
    keys = sum(min(i + 1, WINDOW + KEEP) for i in range(T))
    m._rotations(st, 1, T)
    at = m.attn_args(3, mem.layers[3], st, 0, 1, T, 0, True)
    w3, w0 = m.weights[3], m.weights[0]
    proj = lambda w: m.buf("proj", (w.w_in.shape[0] + 7) // 8 * 8)
    m._gemm(m.x16, w3.w_in, proj(w3), T)
    t.add("layers", "attention (tensor cores)", run(lambda: K.attn_tc(at)), T * (3 * H + 2 * Gq) * hd * 2, 4.0 * keys * H * hd, "attention forward")
    t.add("layers", "rotation + qk norm + cache store", run(lambda: K.qkv_store(at)), T * (H + 2 * Gq) * hd * 4, like="qk norm + rope")
    ma = m.mamba_args(0, mem.layers[0], st, 0, 1, T)
    need = K.ssd_ws_floats(1, ma.H, ma.P, ma.Ns, T)
    if need:
        ma.chunk_ws = m._scratch("ssd", need).data_ptr()
    m._gemm(m.x16, w0.w_in, proj(w0), T)
    n, gn = ma.H * ma.P, ma.G * ma.N
    t.add("layers", "convolution + silu", run(lambda: K.conv(ma)), T * (n + 2 * gn) * 4, like="rmsnorm")
    # per 128-token chunk and head: C B^T and its weights times x (causal halves), C S, the state update
    fl = (T / 128) * ma.H * 2.0 * (128 * 128 * STATE / 2 + 128 * 128 * VDIM / 2 + 2 * 128 * STATE * VDIM)
    t.add("layers", "Mamba-2 chunked recurrence", run(lambda: K.ssd(ma)), T * (2 * n + 2 * gn) * 2, fl, "attention forward")
    t.add("layers", "gated group norm", run(lambda: K.gated_norm(ma)), T * n * 6, like="rmsnorm")
    t.add("layers", "norm of the output + residual add", run(lambda: K.postnorm(m.y, m.x[0], w0.norm1, 1e-5, m.x[0], m.x16, T, d)), T * d * 14, like="rmsnorm")
    t.add("layers", "embedding", run(lambda: K.embed(ids, m.embed, m.x[0], m.x16, d)), T * d * 8, like="embedding")
    t.add("layers", "projection GEMM", run(lambda: m._gemm(m.x16, w0.w_in, proj(w0), T)), 0, 2.0 * T * d * w0.w_in.shape[0], "GEMM")
    t.add("layers", "output GEMM (fp32 out)", run(lambda: m._gemm(m.buf("mixed", w0.w_o.shape[1]), w0.w_o, m.y, T)), 0, 2.0 * T * d * w0.w_o.shape[1], "GEMM (fp32 out + residual)")
    t.add("layers", "gate/up GEMM + SwiGLU", run(lambda: m._mlp_act(w0, T)), 0, 4.0 * T * d * E, "GEMM + SwiGLU")
    dense_prompt_kernels(t, z, ids, T, flush)


def dense_prompt_kernels(t, z, ids, T, flush, full=False):
    """``full``: also the attention without a window."""
    import torch
    from ghassan_b200.ops import gemm as G
    from ghassan_b200.ops import kernels as KK
    d, E, H, Gq, hd = z["width"], z["ff"], z["H"], z["G"], z["hd"]
    f16 = dict(dtype=torch.float16, device="cuda")
    run = lambda fn: time_launch(fn, flush)
    x32, xb, rr = torch.randn(T, d, device="cuda"), torch.zeros(T, d, **f16), torch.zeros(T, device="cuda")
    nw, emb = torch.ones(d, device="cuda"), torch.randn(VOCAB, d, device="cuda")
    t.add("dense", "rmsnorm", run(lambda: KK.rmsnorm_fwd(x32, nw, xb, rr, 1e-5)), T * d * 6)
    t.add("dense", "embedding", run(lambda: KK.embed_fwd(ids, emb, x32)), T * d * 8)
    qd, kvd = H * hd, Gq * hd
    qkv, qk, att, lse = torch.randn(T, qd + 2 * kvd, **f16), torch.zeros(T, qd + kvd, **f16), torch.zeros(T, qd, **f16), torch.zeros(T, H, device="cuda")
    cs = KK.rope_table(torch.linspace(0.001, 1, hd // 2), T, "cuda")
    pos, lo = torch.arange(T, dtype=torch.int32, device="cuda"), torch.zeros(T, dtype=torch.int32, device="cuda")
    qn = torch.ones(hd, device="cuda")
    t.add("dense", "qk norm + rope", run(lambda: KK.qk_norm_rope_fwd(qkv, qk, qn, qn, cs, pos, H, Gq, hd, 1e-5, 0)), T * (H + Gq) * hd * 4)
    dkeys = sum(min(i + 1, WINDOW) for i in range(T))
    t.add("dense", "attention forward", run(lambda: KK.attn_tc_fwd(qk[:, :qd], qk[:, qd:], qkv[:, qd + kvd:], att, lse, None, lo, 1, T, H, Gq, hd, WINDOW,
                                                                   hd ** -0.5)), T * (2 * H + 2 * Gq) * hd * 2, 4.0 * dkeys * H * hd)
    wq, wo = torch.randn(qd + 2 * kvd, d, **f16), torch.randn(d, qd, **f16)
    wgu, act = torch.randn(2 * E, d, **f16), torch.zeros(T, E, **f16)
    t.add("dense", "GEMM", run(lambda: G.gemm(xb, wq, out=qkv)), 0, 2.0 * T * d * (qd + 2 * kvd))
    t.add("dense", "GEMM (fp32 out + residual)", run(lambda: G.gemm(att, wo, out=x32, addend=x32)), 0, 2.0 * T * d * qd)
    t.add("dense", "GEMM + SwiGLU", run(lambda: G.gemm_swiglu(xb, wgu, act_out=act)), 0, 4.0 * T * d * E)
    if full:
        t.add("dense", "attention forward, every token", run(lambda: KK.attn_tc_fwd(qk[:, :qd], qk[:, qd:], qkv[:, qd + kvd:], att, lse, None, lo, 1, T, H, Gq, hd, 0,
                                                                                    hd ** -0.5)), T * (2 * H + 2 * Gq) * hd * 2, 2.0 * T * (T + 1) * H * hd)


def token_kernels(t, z, m, mem, T):
    """One token of one sequence that has seen T."""
    import torch
    from ghassan_b200.ops import decode as D
    from ghassan_b200.ops import kernels as KK
    from ghassan_b200.ops import layers as K
    d, E, H, Gq, hd = z["width"], z["ff"], z["H"], z["G"], z["hd"]
    b16, f16 = dict(dtype=torch.bfloat16, device="cuda"), dict(dtype=torch.float16, device="cuda")
    ctx = torch.tensor([[T - 8, T - 8, 0, 0]], dtype=torch.int32, device="cuda")
    w0 = m.weights[0]
    ma = m.mamba_args(0, mem.layers[0], ctx, 0, 1, 1)
    n = ma.H * ma.P
    y32 = torch.randn(1, d, device="cuda")

    def gemv(label, like, w, f32=False, **kw):
        reps = [w.clone() for _ in range(copies(w.numel() * 2))]
        out = torch.zeros(1, w.shape[0], device="cuda") if f32 else torch.zeros(1, w.shape[0], **b16)
        t.add("layers", label, time_chain([lambda wi=wi: m._gemv(wi, 1, out, **kw) for wi in reps]), w.numel() * 2, like=like)

    res = dict(prologue=1, d=d, x=m.x[0], y=y32, ldy=d, w1=w0.norm1, x_out=m.x[1])
    gv, sq = torch.randn(1, n, device="cuda"), torch.rand(1, 2 * ma.H, device="cuda") * 32
    aa = torch.randn(1, E, **b16)
    gemv("GEMV: projection (norm + add inside)", "GEMV (norm inside)", w0.w_in, **res)
    gemv("GEMV: output (gated norm inside)", "GEMV", w0.w_o, True, prologue=3, d=n, v32=gv, sq=sq, n_sq=2 * ma.H, w1=w0.vec["norm"], parts=z["mg"])
    gemv("GEMV: gate/up + SwiGLU", "GEMV: gate/up + SwiGLU", w0.w_gu, swiglu=1, **res)
    gemv("GEMV: down", "GEMV", w0.w_down, True, prologue=0, d=E, x16=aa, ldx=E)
    gemv("GEMV: vocabulary (both norms inside)", "GEMV: vocabulary", m.head, True, w2=m.final_norm, softcap=30.0, **res)
    cb = 2 * WINDOW * Gq * hd * 2
    kv = [(mem.layers[3].k.clone(), mem.layers[3].v.clone()) for _ in range(16)]

    def at_mk(c):
        a = m.attn_args(3, mem.layers[3], ctx, 0, 1, 1, -1, True)
        a.cache_k, a.cache_v = c[0].data_ptr(), c[1].data_ptr()
        return lambda: K.attn_decode(a)
    t.add("layers", "attention over the cache", time_chain([at_mk(c) for c in kv]), cb, like="attention over the cache")
    a1 = m.attn_args(3, mem.layers[3], ctx, 0, 1, 1, -1, True)
    t.add("layers", "rotation + norm + append", time_chain([lambda: K.qkv_store(a1)] * 20), (H + 2 * Gq) * hd * 4, like="rope + append")
    s_bytes = ma.H * ma.P * ma.Ns * 8

    def st_mk(s):
        a = m.mamba_args(0, mem.layers[0], ctx, 0, 1, 1)
        a.ssm, a.gated, a.gated_sq = s.data_ptr(), gv.data_ptr(), sq.data_ptr()
        return lambda: K.mamba_step(a)
    t.add("layers", "Mamba-2 token step", time_chain([st_mk(mem.layers[0].ssm.clone()) for _ in range(copies(s_bytes))]), s_bytes, like="attention over the cache")
    dense_token_kernels(t, z)


def dense_token_kernels(t, z, contexts=(WINDOW,)):
    import torch
    from ghassan_b200.ops import decode as D
    from ghassan_b200.ops import kernels as KK
    d, E, H, Gq, hd = z["width"], z["ff"], z["H"], z["G"], z["hd"]
    f16 = dict(dtype=torch.float16, device="cuda")
    qd, kvd = H * hd, Gq * hd
    nw, qn = torch.ones(d, device="cuda"), torch.ones(hd, device="cuda")

    def q(N, Kd, k):
        return [D.QWeight(torch.zeros(N * Kd * 2, dtype=torch.uint8, device="cuda"), D.W_F16, N, Kd) for _ in range(k)]
    xx = torch.randn(1, d, device="cuda")
    o16, o32 = torch.zeros(1, max(VOCAB, qd + 2 * kvd), **f16), torch.zeros(1, VOCAB, device="cuda")
    at16, a16 = torch.randn(1, qd, **f16), torch.zeros(1, 1, E, **f16)
    ws = q(qd + 2 * kvd, d, copies((qd + 2 * kvd) * d * 2))
    t.add("dense", "GEMV (norm inside)", time_chain([lambda w=w: D.gemv_norm(w, xx, nw, 1e-5, o16[:, :w.N]) for w in ws]), ws[0].nbytes)
    ws = q(d, qd, copies(d * qd * 2))
    t.add("dense", "GEMV", time_chain([lambda w=w: D.gemv(w, at16, o32[:, :d], addend=xx) for w in ws]), ws[0].nbytes)
    k = copies(4 * E * d)
    ws = list(zip(q(E, d, k), q(E, d, k)))
    t.add("dense", "GEMV: gate/up + SwiGLU", time_chain([lambda w=w: D.swiglu_norm(w[0], w[1], 0, E, d, xx, nw, 1e-5, None, 1, False, a16) for w in ws]), 2 * ws[0][0].nbytes)
    ws = q(VOCAB, d, copies(VOCAB * d * 2))
    t.add("dense", "GEMV: vocabulary", time_chain([lambda w=w: D.gemv_norm(w, xx, nw, 1e-5, o32) for w in ws]), ws[0].nbytes)
    del ws
    for cap in contexts:
        cb = 2 * cap * kvd * 2
        kv = [(torch.randn(1, cap, kvd, **f16), torch.randn(1, cap, kvd, **f16)) for _ in range(copies(cb))]
        sp = torch.arange(cap, dtype=torch.int32, device="cuda").view(1, -1)
        stt = torch.tensor([[cap - 1, cap - 1, 0, 0]], dtype=torch.int32, device="cuda")
        splits = int(min(64, max(8, 512 // Gq)))
        scr = torch.zeros(H * splits * (hd + 2), device="cuda")
        t.add("dense", "attention over the cache" + ("" if cap == WINDOW else ", every token"),
              time_chain([lambda c=c: D.decode_attn(at16, c[0], c[1], sp, stt, o16[:, :qd], scr, splits, H, Gq, hd, cap, 0, hd ** -0.5) for c in kv]), cb)
    qkv1, p1 = torch.randn(1, qd + 2 * kvd, **f16), torch.zeros(1, dtype=torch.int32, device="cuda")
    cs = KK.rope_table(torch.linspace(0.001, 1, hd // 2), 8, "cuda")
    t.add("dense", "rope + append", time_chain([lambda: D.qk_rope_append(qkv1, o16[:, :qd], qn, qn, cs, p1, kv[0][0], kv[0][1], sp, stt, H, Gq, hd, cap, 8, 1e-5, 0)] * 20),
          (H + 2 * Gq) * hd * 4)


def side_prompt_kernels(t, z, m, mem, st, ids, T):
    """Layer 0: window attention, layer 3: latent attention; both with their feed-forward beside them."""
    import torch
    from ghassan_b200.ops import layers as K
    flush = Flush()
    d, E, H, Gq, hd = z["width"], z["ff"], z["H"], z["G"], z["hd"]
    run = lambda fn: time_launch(fn, flush)
    w0, w3, mx = m.weights[0], m.weights[3], m.cfg.layers[3].mixer
    proj = lambda w: m.buf("proj", (w.w_in.shape[0] + 7) // 8 * 8)
    norm = ("layer", w0.norm1, w0.norm1_b)
    m._rotations(st, 1, T)
    m._gemm(m.x16, w0.w_in, proj(w0), T)
    at = m.attn_args(0, mem.layers[0], st, 0, 1, T, 0, True)
    keys = sum(min(i + 1, WINDOW) for i in range(T))
    t.add("side", "attention, capped and biased", run(lambda: K.attn_tc(at)), T * (2 * H + 2 * Gq) * hd * 2, 4.0 * keys * H * hd, "attention forward")
    t.add("side", "query temperature + cache store", run(lambda: K.qkv_store(at)), T * (H + 2 * Gq) * hd * 4, like="qk norm + rope")
    t.add("side", "residual add + layer norm", run(lambda: K.add_norm(m.x[0], T, norm, 1e-5, m.x16, m.y, 0.5, None, m.x[0])), T * d * 14, like="rmsnorm")
    t.add("side", "embedding + layer norm", run(lambda: K.embed_norm(ids, m.embed, ("layer",) + m.embed_norm, 1e-5, m.x0, m.dtype)), T * d * 6, like="embedding")
    t.add("side", "projection GEMM", run(lambda: m._gemm(m.x16, w0.w_in, proj(w0), T)), 0, 2.0 * T * d * w0.w_in.shape[0], "GEMM")
    t.add("side", "up GEMM + squared relu", run(lambda: m._up_rows(0, T)), 0, 2.0 * T * d * E, "GEMM + SwiGLU")
    t.add("side", "output GEMM of both sublayers (fp32 out)", run(lambda: m._gemm(m.mixed(0), w0.w_o, m.y, T)), 0, 2.0 * T * d * w0.w_o.shape[1], "GEMM (fp32 out + residual)")
    m._gemm(m.x16, w3.w_in, proj(w3), T)
    la = m.latent_args(3, mem.layers[3], st, 0, 1, T)
    t.add("side", "latent: projection GEMM", run(lambda: m._gemm(m.x16, w3.w_in, proj(w3), T)), 0, 2.0 * T * d * w3.w_in.shape[0], "GEMM")
    t.add("side", "latent: norms + rotation + cache store", run(lambda: K.latent_store(la)), T * (mx.q_rank + la.ldc) * 4, like="qk norm + rope")
    cq, qc = m.buf("cq", w3.w_uq.shape[1]), m.buf("qc", (w3.w_uq.shape[0] + 7) // 8 * 8)
    t.add("side", "latent: query GEMM", run(lambda: m._gemm(cq, w3.w_uq, qc, T)), 0, 2.0 * T * mx.q_rank * w3.w_uq.shape[0], "GEMM")
    t.add("side", "latent: query rotation", run(lambda: K.latent_queries(la)), T * H * (la.dn + la.dr + la.dkp) * 2, like="qk norm + rope")
    kv, per = m._expanded(3, mem.layers[3], 0, 1, T)
    t.add("side", "latent: key and value GEMM", run(lambda: m._expanded(3, mem.layers[3], 0, 1, T)), 0, 2.0 * T * la.ldc * w3.w_kv.shape[0], "GEMM")
    aa = m.expanded_attn_args(3, la, kv, per, 0)
    t.add("side", "latent: attention", run(lambda: K.attn_tc(aa)), T * H * (2 * la.dkp + 3 * la.dvp) * 2, 1.0 * T * (T + 1) * H * (la.dn + la.dr + la.dv),
          "attention forward, every token")
    dense_prompt_kernels(t, z, ids, T, flush, full=True)


def side_token_kernels(t, z, m, mem, T):
    """One token of one sequence that has seen T."""
    import torch
    from ghassan_b200.ops import layers as K
    d, H, Gq, hd = z["width"], z["H"], z["G"], z["hd"]
    b16 = dict(dtype=torch.bfloat16, device="cuda")
    ctx = torch.tensor([[T - 8, T - 8, 0, 0]], dtype=torch.int32, device="cuda")
    w0, w3, mx = m.weights[0], m.weights[3], m.cfg.layers[3].mixer
    y32 = torch.randn(1, d, device="cuda")
    mixed = m.mixed(0)

    def gemv(label, like, w, f32=False, **kw):
        reps = [w.clone() for _ in range(copies(w.numel() * 2))]
        out = torch.zeros(1, w.shape[0], device="cuda") if f32 else torch.zeros(1, w.shape[0], **b16)
        t.add("side", label, time_chain([lambda wi=wi: m._gemv(wi, 1, out, **kw) for wi in reps]), w.numel() * 2, like=like)

    res = dict(prologue=5, d=d, x=m.x[0], y=y32, ldy=d, alpha=0.5, w1=w0.norm1, b1=w0.norm1_b, norm_mode=1, x_out=m.x[1])
    gemv("GEMV: all input rows (add + norm inside)", "GEMV (norm inside)", w0.w_all, n1=w0.w_in.shape[0], out2=mixed[:, w0.off:], ldo2=mixed.stride(0), **res)
    gemv("GEMV: output of both sublayers", "GEMV", w0.w_o, True, prologue=0, d=w0.w_o.shape[1], x16=mixed, ldx=mixed.stride(0))
    gemv("GEMV: vocabulary (add + norm inside)", "GEMV: vocabulary", m.head, True, **res)
    proj = m.buf("proj", (w3.w_in.shape[0] + 7) // 8 * 8)
    gemv("latent: GEMV queries (norm inside)", "GEMV (norm inside)", w3.w_uq, prologue=4, d=mx.q_rank, x16=proj, ldx=proj.stride(0), w1=w3.vec["dq.norm"])
    c0 = mem.layers[0]
    kv = [(c0.k.clone(), c0.v.clone()) for _ in range(16)]

    def at_mk(c):
        a = m.attn_args(0, c0, ctx, 0, 1, 1, -1, True)
        a.cache_k, a.cache_v = c[0].data_ptr(), c[1].data_ptr()
        return lambda: K.attn_decode(a)
    t.add("side", "attention over the cache", time_chain([at_mk(c) for c in kv]), 2 * WINDOW * Gq * hd * 2, like="attention over the cache")
    a1 = m.attn_args(0, c0, ctx, 0, 1, 1, -1, True)
    t.add("side", "query temperature + append", time_chain([lambda: K.qkv_store(a1)] * 20), (H + 2 * Gq) * hd * 4, like="rope + append")
    m._rotations(ctx, 1, 1)
    maps = [w3.w_kv.clone() for _ in range(copies(w3.w_kv.numel() * 2))]
    rows = [mem.layers[3].rows.clone() for _ in range(copies(mem.layers[3].nbytes))]
    n = max(len(maps), len(rows))

    def la_mk(i, fn):
        a = m.latent_args(3, mem.layers[3], ctx, 0, 1, 1)
        a.W_kv, a.cache = maps[i % len(maps)].data_ptr(), rows[i % len(rows)].data_ptr()
        return lambda: fn(a)
    t.add("side", "latent: queries through the key map + append", time_chain([la_mk(i, lambda a: K.latent_absorb(a, True)) for i in range(n)]),
          H * la_bytes(mx, "dim"), like="GEMV")
    t.add("side", "latent: attention over the latents + value map", time_chain([la_mk(i, K.latent_attn) for i in range(n)]),
          (T - 7) * (mx.kv_rank + mx.rot_dim) * 2 + H * la_bytes(mx, "vdim"), like="attention over the cache, every token")
    dense_token_kernels(t, z, (WINDOW, T))


def la_bytes(mx, side):
    """Bytes of one head's key ("dim") or value ("vdim") map."""
    return getattr(mx, side) * mx.kv_rank * 2


def bench_kernels(name, T, design="zikedra"):
    import torch
    from ghassan_b200.inference.layer_cache import SlotManager
    from ghassan_b200.models.layer_list import random_parameters
    from ghassan_b200.models.layer_model import LayerModel
    z = SIZES[name]
    cfg = layer_config(z, 4) if design == "zikedra" else side_config(name, 4)
    m = LayerModel(cfg, random_parameters(cfg, 1, device="cuda"), 1, T, torch.bfloat16)
    mem = SlotManager(cfg, 1, T, T, torch.bfloat16, m.dev)
    st = torch.zeros(1, 4, dtype=torch.int32, device="cuda")
    ids = torch.randint(0, VOCAB, (T,), dtype=torch.int32, device="cuda")
    mem.claim(0, 1, T)
    m.forward_rows(ids, mem, st, 0, 1, T)
    t = Table(name, T)
    (prompt_kernels if design == "zikedra" else side_prompt_kernels)(t, z, m, mem, st, ids, T)
    torch.cuda.empty_cache()
    (token_kernels if design == "zikedra" else side_token_kernels)(t, z, m, mem, T)


def bench_models(name, T, new, batches, design="zikedra"):
    import torch
    from ghassan_b200.inference.engine import InferenceEngine, SamplingParams
    from ghassan_b200.inference.generator import Generator
    from ghassan_b200.inference.layer_engine import LayerEngine
    from ghassan_b200.models.layer_list import random_parameters
    z = SIZES[name]
    sp = SamplingParams(temperature=0.8, top_k=40, top_p=0.9, min_p=0.0, repetition_penalty=1.0, seed=1)
    for which in ("layers" if design == "zikedra" else "side", "dense"):
        for B in batches:
            Tb = T if B == 1 else 512
            if which != "dense":
                cfg = layer_config(z) if which == "layers" else side_config(name)
                eng = LayerEngine(cfg, random_parameters(cfg, 1, device="cuda"), batch=B, max_len=Tb + new + 8, prefill_chunk=Tb)
            else:
                cfg = dense_config(z)
                eng = InferenceEngine(cfg, random_named(cfg), fmt="f16", batch=B, max_len=Tb + new + 8, prefill_chunk=Tb)
            gen = Generator(eng)
            gen.benchmark(Tb, new, sp)                       # first use: set-up and capture
            r = gen.benchmark(Tb, new, sp)
            print(json.dumps({"size": name, "model": which, "params": cfg.count_parameters(), "batch": B, "prompt_len": Tb, "new_tokens": new,
                              "prefill_tokens_per_s": round(B * Tb / (r["prefill_ms"] / 1e3)), "prefill_ms": round(r["prefill_ms"], 3),
                              "decode_tokens_per_s": round(r["decode_tokens_per_s"], 1), "decode_ms_per_token": round(r["decode_ms_per_token"], 4),
                              "weight_bytes": eng.weight_bytes}), flush=True)
            del eng, gen
            torch.cuda.empty_cache()


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="s,m,l")
    ap.add_argument("--prompt", type=int, default=8192)
    ap.add_argument("--new", type=int, default=128)
    ap.add_argument("--batches", default="1,32")
    ap.add_argument("--design", choices=["zikedra", "dunavik"], default="zikedra")
    ap.add_argument("--only", choices=["kernels", "models"])
    a = ap.parse_args(argv)
    import torch
    from ghassan_b200.utils import log as L
    from bench import ClockSampler
    L.set_log_level(L.WARN)
    torch.manual_seed(0)
    clk = ClockSampler()
    clk.start()
    clk.begin()
    for name in a.sizes.split(","):
        if a.only != "models":
            bench_kernels(name, a.prompt, a.design)
            torch.cuda.empty_cache()
        if a.only != "kernels":
            bench_models(name, a.prompt, a.new, [int(b) for b in a.batches.split(",")], a.design)
    print(json.dumps({"clocks": clk.stop()}), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
