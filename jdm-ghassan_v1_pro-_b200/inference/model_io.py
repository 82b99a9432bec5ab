"""Load a model for inference from any of the supported files (GGUF, legacy .gai, training checkpoint, or a folder with
config.json and safetensors) and build the engine that serves it (tools/inference_cli.cpp:120-260 in the reference does
the same dispatch)."""
from __future__ import annotations

import glob
import json
import os

import numpy as np

from ..formats.loaded import LoadedModel
from ..models import registry
from ..models.layer_list import LayerListConfig


def sniff(path: str) -> str:
    if os.path.isdir(path):
        return "folder" if os.path.exists(os.path.join(path, "config.json")) else "unknown"
    with open(path, "rb") as f:
        magic = f.read(4)
    return {b"GGUF": "gguf", b"GAI1": "gai", b"GKPT": "ckpt"}.get(magic, "unknown")


def load_folder(path: str) -> LoadedModel:
    """A folder with ``config.json``, ``*.safetensors`` and, optionally, ``tokenizer.gtok``."""
    from ..formats import safetensors as ST
    with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as f:
        d = json.load(f)
    cfg = registry.from_json(d).parse(d)
    named = {}
    for part in sorted(glob.glob(os.path.join(glob.escape(path), "*.safetensors"))):
        named.update(ST.load(part))
    if not named:
        raise ValueError(f"{path}: no .safetensors file")
    tok = None
    if os.path.exists(os.path.join(path, "tokenizer.gtok")):
        from ..data.tokenizer import Tokenizer
        tok = Tokenizer.load(os.path.join(path, "tokenizer.gtok"))
    types = sorted({str(t.dtype).replace("torch.", "") for t in named.values()})
    return LoadedModel(cfg, named, [], tok, {"architecture": cfg.architecture, "quant_profile": "+".join(types)}, {}, None)


def load_model(path: str, tokenizer_path: str = "") -> LoadedModel:
    kind = sniff(path)
    if kind == "folder":
        m = load_folder(path)
    elif kind == "gguf":
        from ..formats import gguf as GGUF
        m = GGUF.load_gguf(path)
    elif kind == "gai":
        from ..formats import gai as GAI
        m = GAI.load_gai(path)
    elif kind == "ckpt":
        from ..training import checkpoint as C
        d = C.read(path, with_optimizer=False)
        cfg = C.config_from_dict(d["config"])
        specs = {s.name: s for s in cfg.param_specs()}
        named = {n: np.asarray(a).reshape(specs[n].shape) for n, a in d["params"]}
        m = LoadedModel(cfg, named, [np.asarray(b) for b in d["moe_bias"]], None, {"steps": str(d["state"]["step"])}, {}, None)
    else:
        raise ValueError(f"not a valid model file: {path} (expected .gguf, legacy .gai, a .ckpt or a folder with config.json)")
    if tokenizer_path:
        from ..data.tokenizer import Tokenizer
        m.tokenizer = Tokenizer.load(tokenizer_path)
    return m


def quant_name(m: LoadedModel) -> str:
    md = m.metadata
    for k in ("ghassan.quantization.profile", "quant_profile"):
        v = md.get(k)
        if v:
            return v.decode() if isinstance(v, (bytes, bytearray)) else str(v)
    return "fp32"


def build_engine(m: LoadedModel, batch: int = 1, max_len: int = 2048, fmt: str = "auto", prefill_chunk: int = 1024):
    """Engine whose decode weights keep the file's storage format where the kernels read it directly; on a host without
    a CUDA device the fp32 CPU engine (`cpu_engine.CpuEngine`) over the expanded weights.  Layer-list models run on the
    device only, in bfloat16 (``fmt`` "auto" / "bf16") or true fp32 ("f32")."""
    import torch
    if isinstance(m.cfg, LayerListConfig):
        if not torch.cuda.is_available():
            raise RuntimeError("%s models run on a CUDA device only" % m.cfg.architecture)
        kinds = {"auto": torch.bfloat16, "bf16": torch.bfloat16, "f32": torch.float32}
        if fmt not in kinds:
            raise ValueError("%s models are served as bf16 or f32, not %s" % (m.cfg.architecture, fmt))
        return registry.engine_class(m.cfg)(m.cfg, m.named, batch=batch, max_len=max_len, prefill_chunk=max(prefill_chunk, 2048),
                                            dtype=kinds[fmt])
    if not torch.cuda.is_available():
        from .cpu_engine import CpuEngine
        return CpuEngine(m.cfg, m.named, batch=batch, max_len=min(max_len, max(64, m.cfg.max_seq_len)), moe_bias=m.moe_bias or None)
    InferenceEngine = registry.engine_class(m.cfg)
    raw = m.raw if (m.raw is not None and hasattr(m.raw, "tensor_raw")) else None
    if fmt == "auto" and raw is None:
        fmt = {"int8": "q8_64", "int4": "q4_0"}.get(quant_name(m), "f16")      # .gai block formats
    return InferenceEngine(m.cfg, m.named, fmt=fmt, batch=batch, max_len=min(max_len, max(64, m.cfg.max_seq_len)),
                           prefill_chunk=min(prefill_chunk, max_len), moe_bias=m.moe_bias or None, raw=raw,
                           raw_types=m.tensor_types if raw is not None else None)
