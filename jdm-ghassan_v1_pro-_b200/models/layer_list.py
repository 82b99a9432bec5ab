"""Configuration of models described layer by layer.

A ``config.json`` of this kind names its architecture and lists the layers; each entry has the type of its mixer, the
mixer's sizes and constants, and its feed-forward (or none).  A mixer type is one class in :data:`MIXERS` that reads its
entry, checks it and says which tensors it owns; the engine has the matching kernels.  What a whole design fixes (where its
norms stand and of which kind they are, the feed-forward's activation, parts that every attention layer has) is a
:class:`Design`, found by the architecture's name in :data:`DESIGNS`.  Another design that is a list of such layers is
another entry there and in ``models/registry.py``.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import numpy as np

from ..utils.log import log_warn


def _need(cond, msg):
    if not cond:
        raise ValueError(msg)


def _int(d, key, lo=1, hi=2 ** 31 - 1, default=None):
    v = d.get(key, default)
    _need(isinstance(v, int) and not isinstance(v, bool) and lo <= v <= hi, f"'{key}' must be an integer in [{lo}, {hi}], got {v!r}")
    return v


def _num(d, key, positive=True, default=None):
    v = d.get(key, default)
    _need(isinstance(v, (int, float)) and not isinstance(v, bool) and math.isfinite(v) and (v > 0 or not positive),
          f"'{key}' must be a {'positive ' if positive else ''}number, got {v!r}")
    return float(v)


@dataclass(frozen=True)
class RotaryScaling:
    """Wavelength-dependent slow-down of the rotation: long wavelengths by ``factor``, short ones not at all."""
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class Rotary:
    dims: int                       # leading dimensions of a head that turn
    base: float
    half: bool = False              # pairs (i, i + dims/2) instead of (2i, 2i + 1)
    scaling: Optional[RotaryScaling] = None

    def frequencies(self) -> np.ndarray:
        """Angular frequency per pair, float64 [dims / 2]."""
        i = np.arange(self.dims // 2, dtype=np.float64)
        f = np.power(float(self.base), -2.0 * i / max(1, self.dims))
        s = self.scaling
        if s is None:
            return f
        turns = s.original * f / (2.0 * math.pi)                 # full turns within the original context
        ramp = (turns - s.low) / (s.high - s.low) if s.high != s.low else np.zeros_like(f)
        mixed = (1.0 - ramp) * f / s.factor + ramp * f
        return np.where(turns > s.high, f, np.where(turns < s.low, f / s.factor, mixed))

    @classmethod
    def parse(cls, d: Optional[dict]) -> Optional["Rotary"]:
        if not d:
            return None
        sc = d.get("scaling")
        dims = _int(d, "dims", 0)
        _need(dims % 2 == 0, "'rot.dims' must be even")
        return cls(dims, _num(d, "base"), False,
                   None if not sc else RotaryScaling(_num(sc, "factor"), _num(sc, "low"), _num(sc, "high"), _num(sc, "original")))


@dataclass(frozen=True)
class QueryTemperature:
    """Queries grow with position: times ``1 + coef * ln(floor((p + 1) / every) + 1)``."""
    coef: float
    every: int

    @classmethod
    def parse(cls, d: Optional[dict]) -> Optional["QueryTemperature"]:
        return cls(_num(d, "coef", False), _int(d, "every")) if d else None


@dataclass(frozen=True)
class Design:
    """What all models of an architecture have in common.

    ``block`` "post": sublayers one after the other, each output normed before it joins the residual.  ``block`` "parallel":
    one norm per layer, both sublayers read it, their sum times ``residual_mult`` joins the residual."""
    block: str = "post"
    norm: str = "rms"                # "rms": weight only; "layer": centred, with weight and bias
    embed_norm: bool = False         # the norm stands behind the embedding, too
    activation: str = "swiglu"       # feed-forward: "swiglu" (gate, up, down) or "relu2" (up, down; squared relu)
    qk_norm: bool = True             # attention layers: weightless norm of q and k, soft-max sink, output gate,
    sink: bool = True
    gate: bool = True
    distance_bias: bool = False      # scores less 2^(-8 (h + 1) / heads) per token of distance
    mixers: Tuple[str, ...] = ("attention", "mamba2")


DESIGNS: Dict[str, Design] = {
    "Zikedra": Design(),
    "Dunavik": Design(block="parallel", norm="layer", embed_norm=True, activation="relu2", qk_norm=False, sink=False, gate=False,
                      distance_bias=True, mixers=("attention", "latent_attention")),
}


@dataclass(frozen=True)
class AttentionMixer:
    """Grouped-query attention: rotary positions, an optional weightless RMS norm of q and k, a sliding window that keeps the
    first tokens, a soft-max sink per head, a sigmoid gate on the heads' outputs; or no rotation, tempered queries, capped
    scores and a bias by distance."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Rotary] = None
    window: int = 0                 # 0: every earlier token is visible
    keep_first: int = 0
    qk_norm: bool = True
    sink: bool = True
    gate: bool = True
    q_temp: Optional[QueryTemperature] = None
    softcap: float = 0.0            # score = softcap * tanh(score / softcap)
    distance_bias: bool = False
    kind = "attention"

    @classmethod
    def parse(cls, d: dict, design: Design = Design()) -> "AttentionMixer":
        mask = d.get("mask") or {}
        m = cls(_int(d, "heads"), _int(d, "kv_heads"), _int(d, "dim", 1, 256), _int(d, "vdim", 1, 256), _num(d, "scale", False),
                Rotary.parse(d.get("rot")), _int(mask, "size", 1) if mask.get("size") is not None else 0,
                _int(mask, "keep_first", 0, default=0), design.qk_norm, design.sink, design.gate, QueryTemperature.parse(d.get("q_temp")),
                0.0 if d.get("softcap") is None else _num(d, "softcap"), design.distance_bias)
        _need(m.heads % m.kv_heads == 0, "'heads' must be a multiple of 'kv_heads'")
        _need(m.rot is None or m.rot.dims <= m.dim, "'rot.dims' exceeds 'dim'")
        return m

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    def projection_rows(self) -> List[Tuple[str, int]]:
        """Tensors that read the mixer's input, in the order in which their rows are stacked."""
        rows = [("q", self.heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.kv_heads * self.vdim)]
        return rows + ([("g", self.heads * self.vdim)] if self.gate else [])

    def tensors(self, width: int) -> Dict[str, tuple]:
        t = {n: (r, width) for n, r in self.projection_rows()}
        if self.sink:
            t["sink"] = (self.heads,)
        t["o"] = (width, self.out_features)
        return t


    def slopes(self) -> np.ndarray:
        """Bias per token of distance, by head."""
        return np.power(2.0, -8.0 * np.arange(1, self.heads + 1, dtype=np.float64) / self.heads)


@dataclass(frozen=True)
class LatentAttentionMixer:
    """Attention whose keys and values are linear maps of one normed latent per token (``kv_rank``), with a rotated key part
    (``rot_dim``) that all heads share; queries come from a normed latent of their own (``q_rank``).  Every earlier token is
    visible; the heads' outputs are gated."""
    heads: int
    dim: int                        # unrotated query / key size of a head
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: Optional[Rotary] = None
    kind = "latent_attention"

    @classmethod
    def parse(cls, d: dict, design: Design = Design()) -> "LatentAttentionMixer":
        m = cls(_int(d, "heads"), _int(d, "dim", 1, 256), _int(d, "rot_dim", 1, 256), _int(d, "vdim", 1, 256), _int(d, "kv_rank"), _int(d, "q_rank"),
                _num(d, "scale", False), Rotary.parse(d.get("rot")))
        _need(m.dim + m.rot_dim <= 256, "'dim' + 'rot_dim' must not exceed 256")
        _need(m.kv_rank + m.rot_dim <= 1024, "'kv_rank' + 'rot_dim' must not exceed 1024")
        _need(m.rot is None or m.rot.dims <= m.rot_dim, "'rot.dims' exceeds 'rot_dim'")
        return m

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    def projection_rows(self) -> List[Tuple[str, int]]:
        return [("dq", self.q_rank), ("dkv", self.kv_rank + self.rot_dim), ("g", self.out_features)]

    def tensors(self, width: int) -> Dict[str, tuple]:
        t = {n: (r, width) for n, r in self.projection_rows()}
        t.update({"dq.norm": (self.q_rank,), "uq": (self.heads * (self.dim + self.rot_dim), self.q_rank), "dkv.norm": (self.kv_rank,),
                  "uk": (self.heads * self.dim, self.kv_rank), "uv": (self.out_features, self.kv_rank), "o": (width, self.out_features)})
        return t


@dataclass(frozen=True)
class Mamba2Mixer:
    """State-space mixer with a scalar decay per head, a short causal convolution and a gated norm in equal groups."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int
    kind = "mamba2"

    @classmethod
    def parse(cls, d: dict, design: Design = Design()) -> "Mamba2Mixer":
        m = cls(_int(d, "heads"), _int(d, "vdim"), _int(d, "state", 1, 256), _int(d, "groups"), _int(d, "conv", 1, 32),
                _int(d, "norm_groups", default=1))
        _need(m.heads % m.groups == 0, "'heads' must be a multiple of 'groups'")
        _need(m.out_features % m.norm_groups == 0, "'norm_groups' must divide heads * vdim")
        return m

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.out_features + 2 * self.groups * self.state

    def projection_rows(self) -> List[Tuple[str, int]]:
        return [("in", self.out_features + self.channels + self.heads)]

    def tensors(self, width: int) -> Dict[str, tuple]:
        t = {n: (r, width) for n, r in self.projection_rows()}
        t.update({"conv": (self.channels, self.conv), "conv.b": (self.channels,), "dt_bias": (self.heads,), "A_log": (self.heads,),
                  "D": (self.heads,), "norm": (self.out_features,), "o": (width, self.out_features)})
        return t


MIXERS = {c.kind: c for c in (AttentionMixer, LatentAttentionMixer, Mamba2Mixer)}


@dataclass(frozen=True)
class DenseMlp:
    ff: int
    activation: str = "swiglu"
    kind = "dense"

    @classmethod
    def parse(cls, d: Optional[dict], design: Design = Design()) -> Optional["DenseMlp"]:
        if d is None:
            return None
        _need(d.get("kind", "dense") == "dense", f"unknown feed-forward kind {d.get('kind')!r}")
        return cls(_int(d, "ff"), design.activation)

    def tensors(self, width: int) -> Dict[str, tuple]:
        t = {"gate": (self.ff, width)} if self.activation == "swiglu" else {}
        return dict(t, up=(self.ff, width), down=(width, self.ff))


@dataclass(frozen=True)
class Run:
    """One execution of a layer.  A layer that runs several times has a cache or state per run."""
    layer: int
    rejoin: bool = False            # the embedding output is added to the residual right before it


def layer_runs(n: int, loop: Optional[dict]) -> List[Run]:
    """Order of execution: layers ``start .. stop - 1`` run ``times`` times in a row; every repetition begins with the
    embedding output added once more."""
    if not loop:
        return [Run(i) for i in range(n)]
    a, b, times = _int(loop, "start", 0, n - 1), _int(loop, "stop", 1, n), _int(loop, "times", 1, 4096)
    _need(a < b, "'loop.stop' must lie behind 'loop.start'")
    turns = [Run(i, t > 0 and i == a) for t in range(times) for i in range(a, b)]
    return [Run(i) for i in range(a)] + turns + [Run(i) for i in range(b, n)]


@dataclass(frozen=True)
class LayerSpec:
    mixer: object
    mlp: Optional[DenseMlp]
    weights: int                    # index of the layer whose tensors this one uses (itself, unless shared)


@dataclass
class LayerListConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    eps: float
    layers: List[LayerSpec]
    logit_softcap: float = 0.0
    max_seq_len: int = 65536        # positions are computed, not tabulated: a serving default, not a limit of the model
    extra: dict = field(default_factory=dict)
    design: Design = Design()
    runs: List[Run] = field(default_factory=list)
    residual_mult: float = 1.0

    def __post_init__(self):
        if not self.runs:
            self.runs = layer_runs(len(self.layers), None)

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_json(cls, d: dict) -> "LayerListConfig":
        arch = str(d.get("architecture", ""))
        _need(arch in DESIGNS, f"unknown architecture {arch!r} (known: {', '.join(sorted(DESIGNS))})")
        design = DESIGNS[arch]
        raw = d.get("layers")
        _need(isinstance(raw, list) and raw, "'layers' must be a non-empty list")
        specs: List[LayerSpec] = []
        for i, e in enumerate(raw):
            try:
                kind = e.get("type")
                _need(kind in design.mixers, f"unknown layer type {kind!r} (known: {', '.join(sorted(design.mixers))})")
                own, seen = i, {i}
                while raw[own].get("weights_of") is not None:
                    own = raw[own]["weights_of"]
                    _need(isinstance(own, int) and 0 <= own < len(raw) and own not in seen, "'weights_of' does not lead to a layer with tensors")
                    seen.add(own)
                spec = LayerSpec(MIXERS[kind].parse(e.get("mixer") or {}, design), DenseMlp.parse(e.get("mlp"), design), own)
            except ValueError as err:
                raise ValueError(f"layer {i}: {err}") from None
            specs.append(spec)
        for i, s in enumerate(specs):
            if s.weights != i:
                o = specs[s.weights]
                a, b = ({k: v for k, v in m.tensors(1).items()} for m in (s.mixer, o.mixer))
                _need(type(s.mixer) is type(o.mixer) and a == b and s.mlp == o.mlp,
                      f"layer {i}: shares the tensors of layer {s.weights} but has other sizes")
        cap = d.get("logit_softcap")
        mult = d.get("residual_mult")
        _need(design.block == "parallel" or (mult is None and not d.get("loop")), "'loop' and 'residual_mult' belong to designs with parallel sublayers")
        return cls(arch, _int(d, "vocab"), _int(d, "width"), _num(d.get("norm") or {}, "eps"), specs,
                   0.0 if cap is None else _num(d, "logit_softcap"), design=design, runs=layer_runs(len(specs), d.get("loop")),
                   residual_mult=1.0 if mult is None else _num(d, "residual_mult", False))

    @classmethod
    def from_file(cls, path: str) -> "LayerListConfig":
        with open(path, "r", encoding="utf-8") as f:
            return cls.from_json(json.load(f))

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Every tensor of the model by its name in the file."""
        d = self.hidden_size
        out = {"embed": (self.vocab_size, d)}

        def norm(name):
            out[name] = (d,)
            if self.design.norm == "layer":
                out[name + ".b"] = (d,)

        if self.design.embed_norm:
            norm("embed.norm")
        for i, s in enumerate(self.layers):
            if s.weights != i:
                continue
            p = f"l{i}."
            norm(p + "norm1")
            if s.mlp is not None and self.design.block == "post":
                norm(p + "norm2")
            out.update({p + "mix." + n: sh for n, sh in s.mixer.tensors(d).items()})
            if s.mlp is not None:
                out.update({p + "mlp." + n: sh for n, sh in s.mlp.tensors(d).items()})
        norm("final.norm")
        out["head"] = (self.vocab_size, d)
        return out

    def count_parameters(self) -> int:
        return sum(int(np.prod(s)) for s in self.tensor_shapes().values())

    def summary(self) -> str:
        kinds: Dict[str, int] = {}
        for s in self.layers:
            kinds[s.mixer.kind] = kinds.get(s.mixer.kind, 0) + 1
        shared = sum(1 for i, s in enumerate(self.layers) if s.weights != i)
        return (f"{self.architecture} vocab={self.vocab_size} d={self.hidden_size} L={self.num_layers} ("
                + ", ".join(f"{n} {k}" for k, n in sorted(kinds.items())) + (f", {shared} with shared tensors" if shared else "")
                + (f", {len(self.runs)} runs" if len(self.runs) != self.num_layers else "") + ")"
                + (f" softcap={self.logit_softcap:g}" if self.logit_softcap > 0 else ""))


def check_tensors(cfg: LayerListConfig, named) -> None:
    """Raise when a tensor is missing or has another shape; name what belongs to no layer."""
    want = cfg.tensor_shapes()
    for n, shape in want.items():
        _need(n in named, f"missing tensor '{n}'")
        _need(tuple(named[n].shape) == tuple(shape), f"tensor '{n}' has shape {tuple(named[n].shape)}, expected {tuple(shape)}")
    extra = sorted(set(named) - set(want))
    if extra:
        log_warn("[model] %d tensors belong to no layer and are not used (first: '%s')" % (len(extra), extra[0]))


def random_parameters(cfg: LayerListConfig, seed: int = 0, dtype=None, device="cpu"):
    """Random tensors of the right shapes and sane scales (benchmarks and demonstrations): matrices ~ N(0, 1/in), norms
    around one, decays between slow and fast."""
    import torch
    g = torch.Generator(device=device).manual_seed(seed)
    kw = dict(generator=g, device=device)
    dtype = dtype or torch.bfloat16
    out = {}
    for n, shape in cfg.tensor_shapes().items():
        leaf = n.split(".")[-1] if not n.endswith(".b") else "bias"
        if leaf in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.1 * torch.randn(shape, **kw)
        elif leaf == "A_log":
            t = torch.log(torch.empty(shape, device=device).uniform_(0.5, 8.0, generator=g))
        elif leaf == "dt_bias":
            t = torch.empty(shape, device=device).uniform_(-5.0, -1.0, generator=g)
        elif leaf in ("D", "sink"):
            t = torch.randn(shape, **kw)
        elif leaf == "bias":
            t = 0.1 * torch.randn(shape, **kw)
        elif leaf == "embed":
            t = torch.randn(shape, **kw)
        else:
            t = torch.randn(shape, **kw) * shape[-1] ** -0.5
        out[n] = t.to(dtype)
    return out
