"""Plain implementation of layer-list models (attention, latent attention and Mamba-2 mixers, dense feed-forwards; layers in
sequence or sublayers side by side, with repeated runs of layers): the oracle of ``tests/test_layers_*.py`` and
``tests/test_dunavik_*.py``.

One function per mechanism, written from the equations in double precision, over whole sequences, with the recurrence
as a loop over tokens.  It shares no code with the package: it takes the parsed JSON configuration and a dictionary of
named arrays and knows nothing of caches, portions or kernels.
"""
from __future__ import annotations

import math

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


# ------------------------------------------------------------------------------------------------ rotation
def rotary_frequencies(rot):
    """Angular frequency of every pair, with the wavelength-dependent slow-down where ``scaling`` is given."""
    out = []
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wl = 2.0 * math.pi / f
            if wl > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wl >= sc["original"] / sc["high"]:
                s = (sc["original"] / wl - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return np.array(out)


def rotate(x, rot, positions):
    """x [tokens, heads, dim]: neighbouring dimensions (2i, 2i + 1) below ``dims`` turn by position * frequency."""
    y = np.array(x)
    for i, f in enumerate(rotary_frequencies(rot)):
        a = (np.asarray(positions) * f)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = u * np.cos(a) - v * np.sin(a)
        y[:, :, 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return y


# ------------------------------------------------------------------------------------------------ attention
def visible(i, j, mask):
    """Key j seen from query i: causal, inside the window or among the kept first tokens."""
    return j <= i and (i - j < mask["size"] or j < mask["keep_first"])


def sink_softmax(scores, allowed, sink):
    """Weights of one query: exp(score) over the allowed keys, the sink's exp added to the denominator only."""
    s = np.where(allowed, scores, -np.inf)
    m = max(s.max(), sink)
    e = np.exp(s - m)
    return e / (e.sum() + math.exp(sink - m))


def attention(h, mix, w, eps):
    """h [tokens, width], ``w`` the mixer's tensors by their short names."""
    T = h.shape[0]
    H, G, dk, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = (h @ w["q"].T).reshape(T, H, dk)
    k = (h @ w["k"].T).reshape(T, G, dk)
    v = (h @ w["v"].T).reshape(T, G, dv)
    pos = np.arange(T)
    q, k = rms(rotate(q, mix["rot"], pos), eps), rms(rotate(k, mix["rot"], pos), eps)
    see = np.array([[visible(i, j, mix["mask"]) for j in range(T)] for i in range(T)])
    out = np.zeros((T, H, dv))
    for a in range(H):
        g = a // (H // G)
        sc = (q[:, a] @ k[:, g].T) * mix["scale"]
        for i in range(T):
            out[i, a] = sink_softmax(sc[i], see[i], float(w["sink"][a])) @ v[:, g]
    return (out.reshape(T, H * dv) * sigmoid(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------------------------------------ Mamba-2
def causal_conv(x, kernel, bias):
    """x [tokens, channels], kernel [channels, taps] with the last column on the current token, zeros before."""
    T, taps = x.shape[0], kernel.shape[1]
    xx = np.concatenate([np.zeros((taps - 1, x.shape[1])), x], 0)
    return bias + sum(xx[t0:t0 + T] * kernel[:, t0] for t0 in range(taps))


def ssm(x, B, C, dt, A_log, D, groups):
    """x [T, heads, P], B and C [T, groups, N], dt [T, heads] (already positive): the state recurrence, token by token."""
    T, H, P = x.shape
    S = np.zeros((H, B.shape[2], P))
    y = np.zeros_like(x)
    for t in range(T):
        for a in range(H):
            g = a // (H // groups)
            S[a] = math.exp(-math.exp(A_log[a]) * dt[t, a]) * S[a] + dt[t, a] * np.outer(B[t, g], x[t, a])
            y[t, a] = S[a].T @ C[t, g] + D[a] * x[t, a]
    return y


def gated_group_norm(y, z, weight, parts, eps):
    v = y * silu(z)
    T, n = v.shape
    return rms(v.reshape(T, parts, n // parts), eps).reshape(T, n) * weight


def mamba2(h, mix, w, eps):
    T = h.shape[0]
    H, P, N, G = mix["heads"], mix["vdim"], mix["state"], mix["groups"]
    n = H * P
    p = h @ w["in"].T
    z, xbc, dt = p[:, :n], p[:, n:2 * n + 2 * G * N], p[:, 2 * n + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc[:, :n], xbc[:, n:n + G * N], xbc[:, n + G * N:]
    y = ssm(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w["dt_bias"]), w["A_log"], w["D"], G)
    return gated_group_norm(y.reshape(T, n), z, w["norm"], mix["norm_groups"], eps) @ w["o"].T


# ------------------------------------------------------------------------------------------------ model
def dense_mlp(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"attention": attention, "mamba2": mamba2}


def owner(cfg, i):
    """Index of the layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def run(cfg, weights, tokens, want_layers=False):
    """Logits [tokens, vocab] of one sequence (and the residual after every layer)."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    if cfg["architecture"] == "Dunavik":
        return run_side_by_side(cfg, w, tokens, want_layers)
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    seen = []
    for i, layer in enumerate(cfg["layers"]):
        p = "l%d." % owner(cfg, i)
        x = x + rms(MIXERS[layer["type"]](x, layer["mixer"], sub(w, p + "mix."), eps), eps) * w[p + "norm1"]
        if layer["mlp"] is not None:
            x = x + rms(dense_mlp(x, sub(w, p + "mlp.")), eps) * w[p + "norm2"]
        seen.append(x)
    logits = (rms(x, eps) * w["final.norm"]) @ w["head"].T
    cap = cfg["logit_softcap"]
    logits = cap * np.tanh(logits / cap)
    return (logits, seen) if want_layers else logits


# ------------------------------------------------------------------------------------------------ side by side (Dunavik)
def layer_norm(x, weight, bias, eps):
    """Centred over the last axis, over the root of the mean squared deviation, scaled and shifted."""
    c = x - x.mean(-1, keepdims=True)
    return c / np.sqrt((c * c).mean(-1, keepdims=True) + eps) * weight + bias


def softmax(scores, allowed):
    s = np.where(allowed, scores, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def query_temperature(positions, coef, every):
    """Factor of the query at each position: grows with the logarithm of the number of whole stretches behind it."""
    return np.array([1.0 + coef * math.log((p + 1) // every + 1) for p in positions])


def soft_cap(s, cap):
    return cap * np.tanh(s / cap)


def distance_slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def biased_attention(h, mix, w, eps):
    """Sliding-window attention without rotation: tempered queries, capped scores less a slope times the distance."""
    T = h.shape[0]
    H, G, dk, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = (h @ w["q"].T).reshape(T, H, dk)
    k = (h @ w["k"].T).reshape(T, G, dk)
    v = (h @ w["v"].T).reshape(T, G, dv)
    q = q * query_temperature(range(T), mix["q_temp"]["coef"], mix["q_temp"]["every"])[:, None, None]
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    see = (back >= 0) & (back < mix["mask"]["size"])
    slopes = distance_slopes(H)
    out = np.zeros((T, H, dv))
    for a in range(H):
        g = a // (H // G)
        s = soft_cap((q[:, a] @ k[:, g].T) * mix["scale"], mix["softcap"]) - slopes[a] * back
        out[:, a] = softmax(s, see) @ v[:, g]
    return out.reshape(T, H * dv) @ w["o"].T


def latent_attention(h, mix, w, eps):
    """Queries from a normed latent; keys and values from another one, plus one rotated key part that all heads share."""
    T = h.shape[0]
    H, dn, dr, dv, R = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    pos = np.arange(T)
    q = ((rms(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T).reshape(T, H, dn + dr)
    down = h @ w["dkv"].T
    c = rms(down[:, :R], eps) * w["dkv.norm"]
    k_rot = rotate(down[:, None, R:], mix["rot"], pos)[:, 0]
    q_rot = rotate(q[:, :, dn:], mix["rot"], pos)
    k = (c @ w["uk"].T).reshape(T, H, dn)
    v = (c @ w["uv"].T).reshape(T, H, dv)
    see = pos[None, :] <= pos[:, None]
    out = np.zeros((T, H, dv))
    for a in range(H):
        s = (q[:, a, :dn] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * mix["scale"]
        out[:, a] = softmax(s, see) @ v[:, a]
    return (out.reshape(T, H * dv) * sigmoid(h @ w["g"].T)) @ w["o"].T


def squared_relu_mlp(h, w):
    return np.square(np.maximum(h @ w["up"].T, 0.0)) @ w["down"].T


def layer_runs(cfg):
    """Layers in the order in which they run, with True where the embedding output joins before one."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    turns = [(i, t > 0 and i == a) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, False) for i in range(a)] + turns + [(i, False) for i in range(b, n)]


def run_side_by_side(cfg, w, tokens, want_layers=False):
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    mixers = {"attention": biased_attention, "latent_attention": latent_attention}
    x = first = layer_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], w["embed.norm.b"], eps)
    seen = []
    for i, rejoin in layer_runs(cfg):
        p, layer = "l%d." % i, cfg["layers"][i]
        if rejoin:
            x = x + first
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        y = mixers[layer["type"]](h, layer["mixer"], sub(w, p + "mix."), eps)
        if layer["mlp"] is not None:
            y = y + squared_relu_mlp(h, sub(w, p + "mlp."))
        x = x + mult * y
        seen.append(x)
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
    return (logits, seen) if want_layers else logits
