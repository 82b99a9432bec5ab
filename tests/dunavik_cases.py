"""Small models with side-by-side sublayers for the tests: configurations that share no sizes, weights that make single keys
stand out, and token sequences in which rare tokens ask for others at the edges of what they may see."""
from __future__ import annotations

import copy

import torch

from layers_cases import tokens


def attn(heads, kv, dim, vdim, window, scale=None, cap=25.0, coef=0.4, every=16, mlp=None):
    return {"type": "attention", "mlp": None if mlp is None else {"kind": "dense", "ff": mlp},
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                      "softcap": cap, "mask": {"size": window}, "q_temp": {"coef": coef, "every": every}}}


def latent(heads, dim, rot, vdim, kv_rank, q_rank, scale=None, base=10000.0, mlp=None):
    return {"type": "latent_attention", "mlp": None if mlp is None else {"kind": "dense", "ff": mlp},
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "scale": (dim + rot) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot}}}


def config(layers, width, vocab, loop=None, mult=0.4, eps=1e-5):
    return {"architecture": "Dunavik", "layers": copy.deepcopy(layers), "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))}


def cases():
    """name -> configuration.  Odd sizes, sizes of the tensor-core tiles, and sizes only the general kernels take."""
    return {
        "odd": config([attn(6, 2, 24, 40, 37, cap=12.0, coef=2.0, every=5, mlp=88), latent(3, 20, 10, 28, 44, 36, mlp=130), attn(3, 3, 18, 7, 5),
                       latent(5, 12, 6, 9, 21, 13)], 84, 331, loop=(1, 3, 3), mult=0.3),
        "tiles": config([latent(6, 64, 64, 128, 160, 96, mlp=256), attn(4, 4, 128, 64, 150, cap=40.0, every=100, mlp=136),
                         attn(8, 2, 64, 128, 129, mlp=64)], 160, 200, loop=(0, 2, 2), mult=0.8, eps=1e-3),
        "wide": config([attn(2, 1, 192, 256, 21, cap=80.0, coef=-0.1, every=7), latent(1, 100, 60, 130, 300, 11, mlp=40),
                        latent(7, 30, 34, 64, 70, 300, base=500.0)], 132, 97, mult=1.0),
        "ranks": config([latent(2, 16, 36, 16, 600, 24, mlp=72), attn(5, 5, 64, 64, 1, every=1), attn(1, 1, 8, 8, 400, cap=3.0, mlp=9)], 1100, 150,
                        loop=(2, 3, 1), mult=0.5),
        "temper": config([attn(4, 2, 32, 24, 64, scale=0.06, cap=30.0, coef=5.0, every=9)], 64, 120, mult=1.0),
    }


def weights(cfg, seed=0, match=False):
    """bf16 tensors by name.  ``match``: the query of an even token below 200 is the key of the token after it, so that it
    attends to the places of that token above all others (while the residual is mostly the embedding output)."""
    g = torch.Generator().manual_seed(seed)
    d, out = cfg["width"], {}

    def mat(name, r, c, s=1.0):
        out[name] = torch.randn(r, c, generator=g) * (s * c ** -0.5)

    def vec(name, n, mean=0.0, s=1.0):
        out[name] = mean + s * torch.randn(n, generator=g)

    def norm(name):
        if match:
            out[name], out[name + ".b"] = torch.ones(d), torch.zeros(d)
        else:
            vec(name, d, 1.0, 0.2)
            vec(name + ".b", d, 0.0, 0.3)

    out["embed"] = torch.randn(cfg["vocab"], d, generator=g) * 3.0 + (0.0 if match else 1.0)
    turn = torch.randperm(d, generator=g)
    if match:
        out["embed"][1:200:2] = out["embed"][0:200:2][:, turn]
    norm("embed.norm")
    for i, e in enumerate(cfg["layers"]):
        p, m = "l%d." % i, e["mixer"]
        norm(p + "norm1")
        H, dv = m["heads"], m["vdim"]
        if e["type"] == "attention":
            G, dk = m["kv_heads"], m["dim"]
            mat(p + "mix.q", H * dk, d, 1.5)
            mat(p + "mix.k", G * dk, d, 1.5)
            mat(p + "mix.v", G * dv, d)
            if match:
                k = torch.empty(G * dk, d)
                k[:, turn] = out[p + "mix.k"]                # q(e) = k(e[turn])
                out[p + "mix.q"] = k.view(G, 1, dk, d).expand(G, H // G, dk, d).reshape(H * dk, d).clone()
        else:
            dn, dr, R, Q = m["dim"], m["rot_dim"], m["kv_rank"], m["q_rank"]
            mat(p + "mix.dq", Q, d)
            vec(p + "mix.dq.norm", Q, 1.0, 0.2)
            mat(p + "mix.uq", H * (dn + dr), Q, 2.0)
            mat(p + "mix.dkv", R + dr, d)
            vec(p + "mix.dkv.norm", R, 1.0, 0.2)
            mat(p + "mix.uk", H * dn, R, 2.0)
            mat(p + "mix.uv", H * dv, R, 2.0)
            mat(p + "mix.g", H * dv, d)
            if match:                                        # the query latent of a token is the latent of the token it asks for
                assert Q == R
                out[p + "mix.dq"][:, turn] = out[p + "mix.dkv"][:R]
                out[p + "mix.dq.norm"] = out[p + "mix.dkv.norm"].clone()
                uq = out[p + "mix.uq"].view(H, dn + dr, Q)
                uq[:, :dn] = out[p + "mix.uk"].view(H, dn, R)
                uq[:, dn:] *= 0.3
        mat(p + "mix.o", d, H * dv, 4.0)
        if e["mlp"] is not None:
            mat(p + "mlp.up", e["mlp"]["ff"], d)
            mat(p + "mlp.down", d, e["mlp"]["ff"])
    norm("final.norm")
    mat("head", cfg["vocab"], d, 3.0)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


# A window of 32, and a latent layer that sees everything; one of the layers runs twice.
EDGE_WINDOW, EDGE_EVERY = 32, 24


def edge_case(kind):
    a = attn(4, 2, 24, 32, EDGE_WINDOW, scale=0.3, cap=20.0, coef=0.5, every=EDGE_EVERY, mlp=56)
    b = latent(3, 24, 8, 20, 48, 48, scale=0.11, mlp=40)
    cfg = config([a, b] if kind == "attention" else [b, a], 72, 400, loop=(0, 1, 2), mult=0.25)
    return cfg, weights(cfg, 5, match=True)


def edge_tokens(n=300):
    """(ids, asking places by kind): tokens asked for exactly inside and outside the window, and far behind, on and beside
    the borders of 128-token tiles."""
    ids = tokens({"vocab": 400}, n, 9, lo=200)
    places = {"window_in": [], "window_out": [], "far": []}
    rare = iter(range(0, 200, 2))

    def put(kind, asked, asking):
        assert ids[asked] >= 200 and ids[asking] >= 200
        t = next(rare)
        ids[asked], ids[asking] = t + 1, t
        places[kind].append(asking)

    for p in (60, 95, 129, 165, 190, 287):
        put("window_in", p - (EDGE_WINDOW - 1), p)
    for p in (70, 114, 147, 184, 210, 259):
        put("window_out", p - EDGE_WINDOW, p)
    for asked, asking in ((0, 131), (1, 257), (2, 290), (126, 261), (127, 270), (128, 280), (125, 299)):
        put("far", asked, asking)
    return ids, places
