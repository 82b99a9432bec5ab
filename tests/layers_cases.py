"""Small layer-list models for the tests: configurations that share no sizes, weights that make single keys stand out, and
the distance in which logits are compared."""
from __future__ import annotations

import copy

import numpy as np
import torch


def attn(heads, kv, dim, vdim, window, keep, rot, scale=None, mlp=None, scaling=None, base=10000.0):
    return {"type": "attention", "mlp": None if mlp is None else {"kind": "dense", "ff": mlp},
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                      "mask": {"size": window, "keep_first": keep}, "rot": {"base": base, "dims": rot, "scaling": scaling}}}


def mamba(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mlp": None if mlp is None else {"kind": "dense", "ff": mlp},
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def share(layer, j):
    return dict(copy.deepcopy(layer), weights_of=j)


SCALING = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}


def config(layers, width, vocab, eps=1e-5, cap=20.0):
    return {"architecture": "Zikedra", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap}


def cases():
    """name -> configuration.  Odd sizes, both tensor-core tile widths, and sizes only the general kernels take."""
    a0 = attn(6, 2, 24, 40, 37, 3, 8, mlp=88, scaling=SCALING)
    m0 = mamba(6, 20, 28, 3, 3, 5, mlp=72)
    a1 = attn(4, 4, 128, 64, 150, 130, 32, mlp=130)
    m1 = mamba(3, 96, 128, 1, 4, 1)
    a2 = attn(2, 1, 192, 256, 21, 0, 192)
    m2 = mamba(2, 130, 150, 2, 1, 2, mlp=64)
    a3 = attn(5, 1, 64, 64, 1, 1, 0)
    m3 = mamba(4, 64, 64, 4, 6, 4)
    return {
        "odd": config([a0, m0, share(m0, 1), attn(3, 3, 16, 8, 5, 0, 16), share(a0, 0)], 84, 331),
        "tiles": config([m1, a1, share(m1, 0), mamba(2, 128, 100, 2, 2, 2, mlp=192)], 160, 200, eps=1e-3, cap=7.0),
        "wide": config([a2, m2, a3, m3, share(share(m3, 3), 3)], 132, 97, cap=30.0),
    }


def weights(cfg, seed=0, match=False):
    """bf16 tensors by name, drawn here.  ``match``: the query of an even token below 200 is the key of the token after it,
    so that it attends to the places of that token above all others (in a first layer, where inputs are embeddings)."""
    g = torch.Generator().manual_seed(seed)
    d, out = cfg["width"], {}

    def mat(name, r, c, s=1.0):
        out[name] = torch.randn(r, c, generator=g) * (s * c ** -0.5)

    def vec(name, n, mean=0.0, s=1.0):
        out[name] = mean + s * torch.randn(n, generator=g)

    out["embed"] = torch.randn(cfg["vocab"], d, generator=g)
    turn = torch.randperm(d, generator=g)
    if match:
        out["embed"][1:200:2] = out["embed"][0:200:2][:, turn]
    for i, e in enumerate(cfg["layers"]):
        if e.get("weights_of") is not None:
            continue
        p, m = "l%d." % i, e["mixer"]
        vec(p + "norm1", d, 1.0, 0.2)
        if e["type"] == "attention":
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            mat(p + "mix.q", H * dk, d)
            mat(p + "mix.k", G * dk, d)
            mat(p + "mix.v", G * dv, d)
            mat(p + "mix.g", H * dv, d)
            mat(p + "mix.o", d, H * dv)
            vec(p + "mix.sink", H, 0.5, 1.0)
            if match:
                k = torch.empty(G * dk, d)
                k[:, turn] = out[p + "mix.k"]                # q(e) = k(e[turn])
                k = k.view(G, 1, dk, d)
                out[p + "mix.q"] = k.expand(G, H // G, dk, d).reshape(H * dk, d).clone()
        else:
            n, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            mat(p + "mix.in", 2 * n + 2 * gn + m["heads"], d)
            mat(p + "mix.conv", n + 2 * gn, m["conv"])
            vec(p + "mix.conv.b", n + 2 * gn, 0.0, 0.2)
            vec(p + "mix.dt_bias", m["heads"], -2.0, 1.0)
            out[p + "mix.A_log"] = torch.empty(m["heads"]).uniform_(-2.5, 1.5, generator=g)
            vec(p + "mix.D", m["heads"])
            vec(p + "mix.norm", n, 1.0, 0.2)
            mat(p + "mix.o", d, n)
        if e["mlp"] is not None:
            vec(p + "norm2", d, 1.0, 0.2)
            mat(p + "mlp.gate", e["mlp"]["ff"], d)
            mat(p + "mlp.up", e["mlp"]["ff"], d)
            mat(p + "mlp.down", d, e["mlp"]["ff"])
    vec("final.norm", d, 1.0, 0.2)
    mat("head", cfg["vocab"], d, 3.0)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def as_numpy(w):
    return {k: v.float().numpy() for k, v in w.items()}


def tokens(cfg, n, seed=1, lo=0):
    return np.random.default_rng(seed).integers(lo, cfg["vocab"], n).tolist()


def distance(got, want):
    """Per position: root mean square over the vocabulary of the difference (mean taken off), over the logits' spread."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / want.std()


# A window of 32 behind 5 kept tokens; one attention layer in which an asking token finds one other token.
EDGE_WINDOW, EDGE_KEEP = 32, 5


def edge_case():
    cfg = config([attn(4, 2, 24, 32, EDGE_WINDOW, EDGE_KEEP, 8, scale=0.7, scaling=SCALING), mamba(2, 16, 12, 1, 2, 1)], 64, 400)
    return cfg, weights(cfg, 5, match=True)


def edge_tokens(n=220):
    """Token ids in which rare tokens ask for others that stand exactly inside and outside the edges of the window and of the
    kept prefix, and far behind: (ids, asking places by kind)."""
    ids = tokens({"vocab": 400}, n, 9, lo=200)
    places = {"window_in": [], "window_out": [], "kept_in": [], "kept_out": [], "far": []}
    rare = iter(range(0, 200, 2))

    def put(kind, asked, asking):
        t = next(rare)
        ids[asked], ids[asking] = t + 1, t
        places[kind].append(asking)

    for p in (60, 96, 129, 161, 190):                      # the edge in different places of tiles and portions
        put("window_in", p - (EDGE_WINDOW - 1), p)
    for p in (70, 114, 147, 184, 210):
        put("window_out", p - EDGE_WINDOW, p)
    put("kept_in", EDGE_KEEP - 1, 140)
    put("kept_out", EDGE_KEEP, 150)
    put("far", 2, 215)
    return ids, places
