"""Launchers for the kernels of layer-list models (``csrc/cuda/layers_*.cu``; interface in ``gb_layers.h``)."""
from __future__ import annotations

import ctypes

import torch

from . import _lib

c_int, c_ll, c_vp, c_float = ctypes.c_int, ctypes.c_longlong, ctypes.c_void_p, ctypes.c_float

DTYPE = {torch.bfloat16: 1, torch.float32: 2}
W_FMT = {torch.bfloat16: 1, torch.float32: 6}        # stored-row formats of the GEMV kernels
GEMV_MAX_BATCH = 8
GEMV_MAX_SMEM = 200 * 1024
FINAL_NORM_MAX = 4096                                # widest row whose last norm the GEMV prologue takes along


def head_pad(d: int, dtype) -> int:
    """Row length of a head in q and the caches (zero-padded): whole 128-byte panels for the tensor cores."""
    a = 64 if dtype == torch.bfloat16 else 8
    return (d + a - 1) // a * a


class GemvArgs(ctypes.Structure):
    _fields_ = [
        ("W", c_vp), ("fmt", c_int), ("N", c_int), ("K", c_int),
        ("B", c_int), ("dtype", c_int), ("prologue", c_int), ("swiglu", c_int), ("d", c_int),
        ("x16", c_vp), ("ldx", c_ll),
        ("x", c_vp), ("y", c_vp), ("ldy", c_ll), ("w1", c_vp), ("w2", c_vp), ("eps", c_float), ("x_out", c_vp),
        ("y16", c_vp), ("ldy16", c_ll), ("z16", c_vp), ("ldz", c_ll), ("parts", c_int),
        ("v32", c_vp), ("sq", c_vp), ("n_sq", c_int),
        ("out", c_vp), ("ldo", c_ll), ("out_f32", c_int), ("softcap", c_float),
        ("x0", c_vp), ("alpha", c_float), ("b1", c_vp), ("norm_mode", c_int),
        ("n1", c_int), ("out2", c_vp), ("ldo2", c_ll),
    ]


class AttnArgs(ctypes.Structure):
    _fields_ = [
        ("dtype", c_int), ("B", c_int), ("n", c_int), ("H", c_int), ("G", c_int),
        ("dk", c_int), ("dv", c_int), ("dkp", c_int), ("dvp", c_int),
        ("rot_dims", c_int), ("rot_half", c_int), ("freq", c_vp), ("cs", c_vp), ("qk_norm", c_int), ("eps", c_float), ("scale", c_float),
        ("window", c_int), ("keep", c_int), ("cap", c_int),
        ("proj", c_vp), ("ld_proj", c_ll), ("gate", c_vp), ("ld_gate", c_ll), ("sink", c_vp),
        ("softcap", c_float), ("slopes", c_vp), ("temp_coef", c_float), ("temp_every", c_int),
        ("q", c_vp), ("cache_k", c_vp), ("cache_v", c_vp), ("ld_k", c_ll), ("ld_v", c_ll), ("out", c_vp), ("ldo", c_ll),
        ("scratch", c_vp), ("splits", c_int), ("st", c_vp), ("pos0_max", c_int), ("status", c_vp),
    ]


class LatentArgs(ctypes.Structure):
    _fields_ = [
        ("dtype", c_int), ("B", c_int), ("n", c_int),
        ("H", c_int), ("dn", c_int), ("dr", c_int), ("dv", c_int), ("rank", c_int), ("q_rank", c_int),
        ("dkp", c_int), ("dvp", c_int), ("rot_dims", c_int),
        ("cs", c_vp), ("eps", c_float), ("scale", c_float),
        ("proj", c_vp), ("ld_proj", c_ll), ("q_norm", c_vp), ("kv_norm", c_vp),
        ("cq", c_vp), ("ld_cq", c_ll), ("cache", c_vp), ("ldc", c_int), ("cap", c_int),
        ("qc", c_vp), ("ld_qc", c_ll), ("q", c_vp), ("W_kv", c_vp), ("ld_w", c_ll), ("qa", c_vp),
        ("qa16", c_vp), ("heads_pad", c_int), ("ld_qa16", c_int),
        ("gate", c_vp), ("ld_gate", c_ll), ("out", c_vp), ("ldo", c_ll),
        ("scratch", c_vp), ("splits", c_int), ("st", c_vp), ("status", c_vp),
    ]


class MambaArgs(ctypes.Structure):
    _fields_ = [
        ("dtype", c_int), ("B", c_int), ("n", c_int),
        ("H", c_int), ("P", c_int), ("N", c_int), ("G", c_int), ("taps", c_int), ("Pp", c_int), ("Np", c_int), ("Ns", c_int),
        ("proj", c_vp), ("ld_proj", c_ll),
        ("conv_w", c_vp), ("conv_b", c_vp), ("dt_bias", c_vp), ("A_log", c_vp), ("D", c_vp),
        ("norm_w", c_vp), ("norm_groups", c_int), ("eps", c_float),
        ("conv_state", c_vp), ("ssm", c_vp), ("xh", c_vp), ("bc", c_vp), ("cc", c_vp),
        ("y", c_vp), ("ld_y", c_ll), ("out", c_vp), ("ld_out", c_ll), ("gated", c_vp), ("gated_sq", c_vp),
        ("st", c_vp), ("chunk_ws", c_vp), ("status", c_vp),
    ]


def _p(t):
    return None if t is None else c_vp(t.data_ptr())


def _call(name, *args):
    _lib.check_rc(getattr(_lib.lib(), name)(*args, _lib.stream_ptr()), name)


def embed(ids, table, x, x16, d):
    _call("gb_ll_embed", _p(ids), _p(table), c_ll(table.stride(0)), c_int(table.shape[0]), _p(x), _p(x16), c_ll(x16.stride(0)),
          c_int(ids.numel()), c_int(d), c_int(DTYPE[x16.dtype]))


def postnorm(y, x, w, eps, x_out, x16, rows, d):
    """``x_out = x + y / rms(y) * w`` and its compute-type copy ``x16``."""
    _call("gb_ll_postnorm", _p(y), c_ll(y.stride(0)), _p(x), _p(w), c_float(eps), _p(x_out), _p(x16), c_ll(x16.stride(0)),
          c_int(rows), c_int(d), c_int(DTYPE[x16.dtype]))


def norm_rows(x, row_idx, w, eps, out, rows, d):
    _call("gb_ll_norm_rows", _p(x), _p(row_idx), _p(w), c_float(eps), _p(out), c_ll(out.stride(0)), c_int(rows), c_int(d),
          c_int(DTYPE[out.dtype]))


NORM = {"rms": 0, "layer": 1}


def embed_norm(ids, table, norm, eps, x, dtype):
    """``x = norm(table[ids])``; ``norm``: (kind, weight, bias or None)."""
    kind, w, b = norm
    _call("gb_ll_embed_norm", _p(ids), _p(table), c_ll(table.stride(0)), c_int(table.shape[0]), c_int(NORM[kind]), _p(w), _p(b), c_float(eps),
          _p(x), c_int(ids.numel()), c_int(x.shape[1]), c_int(DTYPE[dtype]))


def add_norm(x, rows, norm=None, eps=0.0, out=None, y=None, alpha=1.0, x0=None, x_out=None, row_idx=None):
    """``v = x + alpha * y + x0``; ``x_out = v`` and ``out = norm(v)`` in the compute type, each where it is asked for."""
    kind, w, b = norm if norm is not None else ("rms", None, None)
    _call("gb_ll_add_norm", _p(y), c_ll(0 if y is None else y.stride(0)), c_float(alpha), _p(x), _p(x0), _p(row_idx), c_int(NORM[kind]), _p(w), _p(b),
          c_float(eps), _p(x_out), _p(out), c_ll(0 if out is None else out.stride(0)), c_int(rows), c_int(x.shape[1]),
          c_int(1 if out is None else DTYPE[out.dtype]))


def relu2_f32(v, rows, n):
    _call("gb_ll_relu2_f32", _p(v), c_ll(v.stride(0)), c_int(rows), c_int(n))


def softcap(v, rows, n, cap):
    _call("gb_ll_softcap", _p(v), c_ll(v.stride(0)), c_int(rows), c_int(n), c_float(cap))


def gemm_f32(a, b, out, rows):
    """``out[:rows] = a[:rows] @ b^T`` with fp32 products (no reduced-precision mode)."""
    _call("gb_ll_gemm_f32", _p(a), c_ll(a.stride(0)), _p(b), c_ll(b.stride(0)), _p(out), c_ll(out.stride(0)), c_int(rows),
          c_int(b.shape[0]), c_int(b.shape[1]))


def swiglu_f32(gu, act, rows, E):
    _call("gb_ll_swiglu_f32", _p(gu), c_ll(gu.stride(0)), _p(act), c_ll(act.stride(0)), c_int(rows), c_int(E))


def advance(state, pos_out, n):
    _call("gb_ll_advance", _p(state), _p(pos_out), c_int(state.shape[0]), c_int(n))


def gemv(a: GemvArgs):
    _call("gb_ll_gemv", ctypes.byref(a))


def rotations(freq, state, B, n, cs):
    """Cosines and sines of ``n`` consecutive positions of each sequence: ``cs`` [B * n, pairs, 2]."""
    _call("gb_ll_rotations", _p(freq), c_int(freq.numel()), _p(state), c_int(B), c_int(n), _p(cs))


def qkv_store(a: AttnArgs):
    _call("gb_ll_qkv_store", ctypes.byref(a))


def attn_prefill(a: AttnArgs):
    _call("gb_ll_attn_prefill", ctypes.byref(a))


def attn_tc_ok(a: AttnArgs) -> bool:
    return _lib.lib().gb_ll_attn_tc_ok(ctypes.byref(a)) == 0


def attn_tc(a: AttnArgs):
    _call("gb_ll_attn_tc", ctypes.byref(a))


def attn_decode(a: AttnArgs):
    _call("gb_ll_attn_decode", ctypes.byref(a))


def latent_store(a: LatentArgs):
    _call("gb_ll_latent_store", ctypes.byref(a))


def latent_queries(a: LatentArgs):
    _call("gb_ll_latent_queries", ctypes.byref(a))


def latent_absorb(a: LatentArgs, store: bool):
    _call("gb_ll_latent_absorb", ctypes.byref(a), c_int(int(store)))


def latent_tc_plan(a: LatentArgs):
    """(heads_pad, ld_qa16) of the tensor-core kernel, or None when it does not cover the shapes."""
    hp, ld = c_int(0), c_int(0)
    return (hp.value, ld.value) if _lib.lib().gb_ll_latent_tc_plan(ctypes.byref(a), ctypes.byref(hp), ctypes.byref(ld)) == 0 else None


def latent_attn(a: LatentArgs):
    _call("gb_ll_latent_attn", ctypes.byref(a))


def conv(a: MambaArgs):
    _call("gb_ll_conv", ctypes.byref(a))


def scan(a: MambaArgs):
    _call("gb_ll_scan", ctypes.byref(a))


def ssd_ok(a: MambaArgs) -> bool:
    return _lib.lib().gb_ll_ssd_ok(ctypes.byref(a)) == 0


def ssd_ws_floats(B, H, P, Ns, n, segments=0) -> int:
    f = _lib.lib().gb_ll_ssd_ws_floats
    f.restype = c_ll
    return int(f(c_int(B), c_int(H), c_int(P), c_int(Ns), c_int(n), c_int(segments)))


def ssd(a: MambaArgs, segments=0):
    """The recurrence in chunks on the tensor cores; ``segments``: runs a sequence is cut into (0: by the machine)."""
    _lib.check_rc(_lib.lib().gb_ll_ssd(ctypes.byref(a), c_int(segments), _lib.stream_ptr()), "gb_ll_ssd")


def mamba_step(a: MambaArgs):
    _call("gb_ll_mamba_step", ctypes.byref(a))


def gated_norm(a: MambaArgs):
    _call("gb_ll_gated_norm", ctypes.byref(a))
