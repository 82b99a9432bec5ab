"""Layer-list models on the device against the plain oracle: every mechanism alone, whole prompts, portions, decoding,
batches, slots that are used again, and generation through the framework's own entry points."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import layers_cases as C
import layers_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

BF, F32 = torch.bfloat16, torch.float32
LIMIT = {BF: 0.08, F32: 3e-5}            # distance of logits; a planted mistake moves them by 0.2 and more
DTYPES = [F32, BF]
_oracle = {}


def engine(raw, w, dtype, **kw):
    from ghassan_b200.inference.layer_engine import LayerEngine
    from ghassan_b200.models.layer_list import LayerListConfig
    return LayerEngine(LayerListConfig.from_json(raw), w, dtype=dtype, **kw)


def case(name, n=300, seed=0):
    raw = C.cases()[name]
    w = C.weights(raw, seed)
    ids = C.tokens(raw, n, seed + {"odd": 16, "wide": 15, "tiles": 17}[name])      # no token whose mixer output nearly cancels
    key = (name, n, seed)
    if key not in _oracle:
        _oracle[key] = O.run(raw, C.as_numpy(w), ids)
    return raw, w, ids, _oracle[key]


def feed(eng, key, ids, cuts):
    """All logits of ``ids`` given in portions that end at ``cuts``."""
    out, lo = [], 0
    for hi in list(cuts) + [len(ids)]:
        if hi > lo:
            out.append(eng.step(key, ids[lo:hi], range(hi - lo)).cpu().numpy())
            lo = hi
    eng.check()
    return np.concatenate(out)


# ------------------------------------------------------------------------------------------------ whole prompts and portions
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(C.cases()))
def test_whole_prompt(name, dtype):
    raw, w, ids, want = case(name)
    d = C.distance(feed(engine(raw, w, dtype), "a", ids, []), want)
    assert d.max() < LIMIT[dtype], (d.max(), int(d.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(C.cases()))
def test_token_by_token(name, dtype):
    raw, w, ids, want = case(name)
    d = C.distance(feed(engine(raw, w, dtype), "a", ids, range(1, len(ids))), want)
    assert d.max() < LIMIT[dtype], (d.max(), int(d.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(C.cases()))
@pytest.mark.parametrize("cuts", [(2, 4, 7, 8, 129, 131, 299), tuple(range(2, 300, 2)), (40, 80, 81, 200), (128, 256), (17, 34, 161)])
def test_portions(name, dtype, cuts):
    raw, w, ids, want = case(name)
    d = C.distance(feed(engine(raw, w, dtype), "a", ids, cuts), want)
    assert d.max() < LIMIT[dtype], (d.max(), int(d.argmax()))


@pytest.mark.parametrize("name", sorted(C.cases()))
def test_prompts_longer_than_a_pass_are_cut_inside(name):
    raw, w, ids, want = case(name)
    eng = engine(raw, w, F32, prefill_chunk=37, max_len=4000)
    assert C.distance(feed(eng, "a", ids, []), want).max() < LIMIT[F32]


@pytest.mark.parametrize("name", sorted(C.cases()))
def test_tensor_core_kernels_and_general_kernels_agree(name):
    raw, w, ids, _ = case(name)
    a = feed(engine(raw, w, BF), "a", ids, [190])
    b = feed(engine(raw, w, BF, use_tensor_cores=False), "a", ids, [190])
    assert C.distance(a, b).max() < LIMIT[BF]


@pytest.mark.parametrize("name", sorted(C.cases()))
def test_residual_after_every_layer(name):
    raw, w, ids, _ = case(name)
    want = O.run(raw, C.as_numpy(w), ids, True)[1]
    eng = engine(raw, w, F32)
    s = eng.mem.acquire("a")
    seen = []
    eng._rows(torch.tensor(ids, dtype=torch.int32, device="cuda"), s, 1, len(ids), lambda i, x: seen.append(x.cpu().numpy()))
    for i, (a, b) in enumerate(zip(seen, want)):
        assert np.abs(a - b).max() < 2e-5 * np.abs(b).max(), i


# ------------------------------------------------------------------------------------------------ edges
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [(), tuple(range(1, 220)), (59, 60, 61, 95, 128, 130, 143), (5, 6, 96, 97, 112, 140, 176), tuple(range(3, 220, 3))])
def test_window_edges_kept_tokens_and_far_keys(dtype, cuts):
    raw, w = C.edge_case()
    ids, places = C.edge_tokens()
    want = O.run(raw, C.as_numpy(w), ids)
    d = C.distance(feed(engine(raw, w, dtype), "a", ids, cuts), want)
    assert d.max() < LIMIT[dtype], {k: d[v].max() for k, v in places.items()}


def _edge_layer(window, keep, n, dim=64, vdim=64, heads=2, kv=1, rot=16, scale=0.4):
    """One attention layer with inputs in which query ``i`` singles out key ``j`` for planted pairs."""
    return C.config([C.attn(heads, kv, dim, vdim, window, keep, rot, scale=scale)], 64, 400)


@pytest.mark.parametrize("window, keep, vdim", [(128, 0, 64), (129, 1, 128), (300, 130, 64), (257, 128, 128), (1, 3, 64)])
def test_tensor_core_attention_at_tile_edges(window, keep, vdim):
    """Windows and kept prefixes on and beside tile borders, long prompts cut at awkward places, a ring that wraps."""
    raw = _edge_layer(window, keep, 900, vdim=vdim)
    w = C.weights(raw, 3, match=True)
    ids = C.tokens(raw, 900, 4, lo=200)
    rare = iter(range(0, 200, 2))
    for p in (450, 513, 641, 768, 895):
        for back in (window - 1, window, max(0, p - keep), max(0, p - keep + 1)):
            if 0 < back <= p and ids[p - back] >= 200:
                t = next(rare)
                ids[p - back], ids[p] = t + 1, t
                break
    want = O.run(raw, C.as_numpy(w), ids)
    for cuts in ((), (1, 300, 301, 640), (257, 512, 770)):
        eng = engine(raw, w, BF, max_len=900, prefill_chunk=400)
        d = C.distance(feed(eng, "a", ids, cuts), want)
        assert d.max() < LIMIT[BF], (cuts, d.max(), int(d.argmax()))
        assert C.distance(feed(engine(raw, w, F32, max_len=900, prefill_chunk=400), "a", ids, cuts), want).max() < LIMIT[F32]


# ------------------------------------------------------------------------------------------------ mechanisms alone
def _one_layer(layer, width=64, dtype=F32, slots=1, rows=512, seed=0):
    """A model of one layer and its memory, for kernels on hand-made projections."""
    from ghassan_b200.inference.layer_cache import SlotManager
    from ghassan_b200.models.layer_list import LayerListConfig
    from ghassan_b200.models.layer_model import LayerModel
    raw = C.config([layer], width, 32)
    cfg = LayerListConfig.from_json(raw)
    m = LayerModel(cfg, C.weights(raw, seed), slots, rows, dtype)
    mem = SlotManager(cfg, slots, 4096, rows, dtype, m.dev)
    state = torch.zeros(slots, 4, dtype=torch.int32, device="cuda")
    return raw, m, mem, state


def _mamba_inputs(m, rows, seed, dt_shift=0.0):
    mx = m.cfg.layers[0].mixer
    n = m.weights[0].w_in.shape[0]
    buf = m.buf("proj", (n + 7) // 8 * 8)
    g = torch.Generator().manual_seed(seed)
    x = torch.randn(rows, n, generator=g)
    x[:, n - mx.heads:] += dt_shift
    buf[:rows, :n] = x.to(buf.dtype).cuda()
    return buf[:rows, :n].float().cpu().double().numpy()


def _mamba_reference(m, proj, start=0, S0=None):
    """Convolved x, B, C as the device rounds them, and the recurrence on them."""
    mx, v = m.cfg.layers[0].mixer, {k: t.cpu().double().numpy() for k, t in m.weights[0].vec.items()}
    n, gn, T = mx.out_features, mx.groups * mx.state, proj.shape[0]
    xbc = O.silu(O.causal_conv(proj[:, n:2 * n + 2 * gn], v["conv"], v["conv.b"]))
    if m.dtype == BF:
        xbc = torch.from_numpy(xbc).to(BF).double().numpy()
    x, B, Cc = (xbc[:, a:b] for a, b in ((0, n), (n, n + gn), (n + gn, n + 2 * gn)))
    dt = O.softplus(proj[:, 2 * n + 2 * gn:] + v["dt_bias"])
    y = O.ssm(x.reshape(T, mx.heads, mx.vdim), B.reshape(T, mx.groups, -1), Cc.reshape(T, mx.groups, -1), dt, v["A_log"], v["D"], mx.groups)
    return xbc, y.reshape(T, n)


def _final_state(m, proj):
    """State after the last token, from the recurrence on device-rounded inputs."""
    mx, v = m.cfg.layers[0].mixer, {k: t.cpu().double().numpy() for k, t in m.weights[0].vec.items()}
    xbc, _ = _mamba_reference(m, proj)
    n, gn, T = mx.out_features, mx.groups * mx.state, proj.shape[0]
    x = xbc[:, :n].reshape(T, mx.heads, mx.vdim)
    B = xbc[:, n:n + gn].reshape(T, mx.groups, -1)
    dt = O.softplus(proj[:, 2 * n + 2 * gn:] + v["dt_bias"])
    S = np.zeros((mx.heads, mx.vdim, mx.state))
    for t in range(T):
        for h in range(mx.heads):
            S[h] = np.exp(-np.exp(v["A_log"][h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(x[t, h], B[t, h // (mx.heads // mx.groups)])
    return S


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7, 12])
def test_convolution_and_its_carried_inputs(dtype, taps):
    from ghassan_b200.ops import layers as K
    raw, m, mem, state = _one_layer(C.mamba(3, 20, 12, 3, taps, 1), dtype=dtype)
    mx = m.cfg.layers[0].mixer
    proj = _mamba_inputs(m, 150, 2)
    want, _ = _mamba_reference(m, proj)
    src = m.buf("proj", (m.weights[0].w_in.shape[0] + 7) // 8 * 8)
    whole = src[:150].clone()
    lo = 0
    for n in (1, 2, 30, 1, 60, 3, 53):
        src[:n] = whole[lo:lo + n]
        a = m.mamba_args(0, mem.layers[0], state, 0, 1, n)
        K.conv(a)
        x = m.buf("xh20x12", mx.heads * a.Pp)[:n].view(n, mx.heads, a.Pp)[..., :20].reshape(n, -1)
        b, c = (m.buf(s + "20x12", mx.groups * a.Np)[:n].view(n, mx.groups, a.Np)[..., :12].reshape(n, -1) for s in ("bc", "cc"))
        got = torch.cat([x, b, c], 1).float().cpu().numpy()
        ref = want[lo:lo + n]
        assert np.abs(got - ref).max() < (1e-5 if dtype == F32 else 2.0 ** -7) * max(1.0, np.abs(ref).max()), (taps, lo)
        state[:, 0] += n
        lo += n


@pytest.mark.parametrize("P, N, heads, groups", [(64, 128, 4, 1), (20, 28, 6, 3), (128, 100, 2, 2), (96, 64, 3, 1), (130, 150, 2, 2), (7, 5, 4, 2)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_token_recurrence(dtype, P, N, heads, groups):
    from ghassan_b200.ops import layers as K
    raw, m, mem, state = _one_layer(C.mamba(heads, P, N, groups, 3, 1), dtype=dtype)
    proj = _mamba_inputs(m, 70, 3)
    _, want = _mamba_reference(m, proj)
    a = m.mamba_args(0, mem.layers[0], state, 0, 1, 70)
    K.conv(a)
    K.scan(a)
    got = m.buf("ssm_y", heads * P)[:70].float().cpu().numpy()
    tol = 2e-5 if dtype == F32 else 2.0 ** -7
    assert np.abs(got - want).max() < tol * np.abs(want).max()
    S = mem.layers[0].ssm[0, :, :, :N].cpu().numpy()
    ref = _final_state(m, proj)
    assert np.abs(S - ref).max() < (1e-5 if dtype == F32 else 1e-2) * np.abs(ref).max()


@pytest.mark.parametrize("P, N, heads, groups", [(64, 128, 4, 1), (20, 28, 6, 3), (128, 100, 2, 2), (96, 64, 3, 1)])
@pytest.mark.parametrize("n, segments", [(128, 1), (400, 1), (400, 2), (390, 4), (129, 2), (77, 0), (512, 0)])
def test_chunked_recurrence(P, N, heads, groups, n, segments):
    """Outputs to one rounding, the carried state to fp32 accuracy of its two-term operands, for slow and fast decays."""
    from ghassan_b200.ops import layers as K
    raw, m, mem, state = _one_layer(C.mamba(heads, P, N, groups, 4, 1), dtype=BF)
    m.weights[0].vec["A_log"].copy_(torch.linspace(-6.0, 3.0, heads))
    proj = _mamba_inputs(m, n, 4, dt_shift=1.0)
    a = m.mamba_args(0, mem.layers[0], state, 0, 1, n)
    assert K.ssd_ok(a)
    need = K.ssd_ws_floats(1, heads, P, a.Ns, n, segments)
    if need:
        ws = torch.full((need,), float("nan"), device="cuda")
        a.chunk_ws = ws.data_ptr()
    K.conv(a)
    K.ssd(a, segments)
    from ghassan_b200.ops import _lib
    _lib.check_status(m.dev)
    got = m.buf("ssm_y", heads * P)[:n].float().cpu().numpy()
    S = mem.layers[0].ssm[0, :, :, :N].cpu().numpy()
    K.scan(a)                                               # the same inputs through the token-by-token kernel
    y2, S2 = m.buf("ssm_y", heads * P)[:n].float().cpu().numpy(), mem.layers[0].ssm[0, :, :, :N].cpu().numpy()
    for h in range(heads):
        ref = np.abs(S2[h]).max()
        assert np.abs(S[h] - S2[h]).max() < 1e-4 * ref, (h, np.abs(S[h] - S2[h]).max() / ref)
        c = slice(h * P, (h + 1) * P)
        assert np.abs(got[:, c] - y2[:, c]).max() < 2.0 ** -7 * np.abs(y2[:, c]).max(), h
    _, want = _mamba_reference(m, proj)
    assert np.abs(got - want).max() < 2.0 ** -5 * np.abs(want).max()


@pytest.mark.parametrize("P, N", [(64, 128), (20, 28), (128, 100)])
def test_chunked_recurrence_continues_from_a_state(P, N):
    from ghassan_b200.ops import layers as K
    raw, m, mem, state = _one_layer(C.mamba(2, P, N, 1, 4, 1), dtype=BF)
    m.weights[0].vec["A_log"].copy_(torch.tensor([-5.0, -3.0]))
    src = m.buf("proj", (m.weights[0].w_in.shape[0] + 7) // 8 * 8)
    _mamba_inputs(m, 500, 5)
    whole = src[:500].clone()
    y = torch.zeros(500, 2 * P, device="cuda")
    ref_mem = torch.zeros_like(mem.layers[0].ssm)
    for kernel in ("scan", "ssd"):
        state.zero_()
        lo = 0
        for n in (130, 5, 128, 200, 37):
            src[:n] = whole[lo:lo + n]
            a = m.mamba_args(0, mem.layers[0], state, 0, 1, n)
            ws = torch.empty(max(1, K.ssd_ws_floats(1, 2, P, a.Ns, n, 2)), device="cuda")
            a.chunk_ws = ws.data_ptr()
            K.conv(a)
            K.scan(a) if kernel == "scan" else K.ssd(a, 2)
            got = m.buf("ssm_y", 2 * P)[:n].float()
            if kernel == "scan":
                y[lo:lo + n] = got
            else:
                assert float((got - y[lo:lo + n]).abs().max()) < 2.0 ** -7 * float(y.abs().max()), (lo, n)
            state[:, 0] += n
            lo += n
        if kernel == "scan":
            ref_mem.copy_(mem.layers[0].ssm)
    assert float((mem.layers[0].ssm - ref_mem).abs().max()) < 1e-4 * float(ref_mem.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_token_step_equals_the_portion_kernels(dtype):
    from ghassan_b200.ops import layers as K
    out = {}
    for step in (False, True):
        raw, m, mem, state = _one_layer(C.mamba(6, 40, 36, 2, 4, 3), dtype=dtype)
        src = m.buf("proj", (m.weights[0].w_in.shape[0] + 7) // 8 * 8)
        _mamba_inputs(m, 40, 6)
        whole, ys = src[:40].clone(), []
        for t in range(40):
            src[:1] = whole[t:t + 1]
            a = m.mamba_args(0, mem.layers[0], state, 0, 1, 1)
            if step:
                K.mamba_step(a)
            else:
                K.conv(a)
                K.scan(a)
            ys.append(m.buf("ssm_y", 240)[:1].float().clone())
            state[:, 0] += 1
        out[step] = (torch.cat(ys), mem.layers[0].ssm.clone(), mem.layers[0].conv.clone())
    for a, b in zip(out[False], out[True]):
        assert float((a.float() - b.float()).abs().max()) <= 1e-6 * float(a.float().abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("parts, P", [(1, 20), (2, 50), (6, 30), (12, 36), (1, 1500)])
def test_gated_group_norm(dtype, parts, P):
    from ghassan_b200.ops import layers as K
    heads = 6
    raw, m, mem, state = _one_layer(C.mamba(heads, P, 8, 1, 2, parts), dtype=dtype, rows=16)
    proj = _mamba_inputs(m, 9, 7)
    y = m.buf("ssm_y", heads * P)
    y[:9] = torch.randn(9, heads * P, generator=torch.Generator().manual_seed(1)).to(dtype).cuda()
    a = m.mamba_args(0, mem.layers[0], state, 0, 1, 9)
    K.gated_norm(a)
    got = m.buf("mixed", m.weights[0].w_o.shape[1])[:9, :heads * P].float().cpu().numpy()
    want = O.gated_group_norm(y[:9].double().cpu().numpy(), proj[:, :heads * P], m.weights[0].vec["norm"].cpu().double().numpy(), parts, m.cfg.eps)
    assert np.abs(got - want).max() < (3e-6 if dtype == F32 else 2.0 ** -8) * np.abs(want).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim, rot, pos", [(24, 8, 0), (64, 64, 1000), (128, 32, 70000), (20, 0, 5), (256, 200, 12345)])
def test_rotation_and_query_key_norm(dtype, dim, rot, pos):
    from ghassan_b200.ops import layers as K
    layer = C.attn(3, 1, dim, 16, 50, 2, rot, scaling=C.SCALING)
    raw, m, mem, state = _one_layer(layer, dtype=dtype)
    n = 5
    src = m.buf("proj", (m.weights[0].w_in.shape[0] + 7) // 8 * 8)
    src[:n] = torch.randn(n, src.shape[1], generator=torch.Generator().manual_seed(3)).to(dtype).cuda()
    proj = src[:n].double().cpu().numpy()
    state[:, 0] = pos
    a = m.attn_args(0, mem.layers[0], state, 0, 1, n, -1)
    K.qkv_store(a)
    p = np.arange(pos, pos + n)
    q = O.rms(O.rotate(proj[:, :3 * dim].reshape(n, 3, dim), layer["mixer"]["rot"], p), m.cfg.eps)
    k = O.rms(O.rotate(proj[:, 3 * dim:4 * dim].reshape(n, 1, dim), layer["mixer"]["rot"], p), m.cfg.eps)
    tol = 2e-6 if dtype == F32 else 2.0 ** -8
    gq = m.buf("q", 3 * a.dkp)[:n].view(n, 3, a.dkp)
    assert np.abs(gq[..., :dim].float().cpu().numpy() - q).max() < tol * np.abs(q).max()
    assert float(gq[..., dim:].abs().sum()) == 0.0
    c = mem.layers[0]
    rows = [x if x < c.keep else c.keep + (x - c.keep) % (c.cap - c.keep) for x in p]
    assert np.abs(c.k[0, rows, :, :dim].float().cpu().numpy() - k).max() < tol * np.abs(k).max()
    assert np.abs(c.v[0, rows, 0, :16].float().cpu().numpy() - proj[:, 4 * dim:4 * dim + 16]).max() == 0.0


def test_fp32_product_is_true_fp32():
    from ghassan_b200.ops import layers as K
    g = torch.Generator().manual_seed(0)
    for M, N, Kd in ((1, 5, 8), (70, 130, 72), (257, 64, 1000)):
        a, b = torch.randn(M, Kd, generator=g).cuda(), torch.randn(N, Kd, generator=g).cuda()
        out = torch.zeros(M, N, device="cuda")
        K.gemm_f32(a, b, out, M)
        ref = a.double() @ b.double().t()
        assert float((out.double() - ref).abs().max()) < 1e-6 * Kd ** 0.5 * 8


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [1, 3, 8])
@pytest.mark.parametrize("d, N", [(36, 50), (300, 333), (2100, 70), (5000, 24)])
def test_gemv_prologues(dtype, B, d, N):
    """Residual add with the norm of the sublayer's output, the last norm, the gated group norm, SwiGLU and the cap."""
    from ghassan_b200.ops import layers as K
    g = torch.Generator().manual_seed(d + N)
    Kp = (d + 7) // 8 * 8
    E = (N + 63) // 64 * 64
    w = torch.zeros(2 * E, Kp, dtype=dtype, device="cuda")
    w[:, :d] = (torch.randn(2 * E, d, generator=g) * d ** -0.5).to(dtype).cuda()
    x, y = (torch.randn(B, d, generator=g).cuda() for _ in range(2))
    w1, w2 = (1 + 0.1 * torch.randn(d, generator=g).cuda() for _ in range(2))
    tol = 1e-5 if dtype == F32 else 2.0 ** -6

    def run(n_rows, out, **kw):
        a = K.GemvArgs()
        a.W, a.fmt, a.N, a.K, a.B, a.dtype, a.d, a.eps = w.data_ptr(), K.W_FMT[dtype], n_rows, Kp, B, K.DTYPE[dtype], d, 1e-4
        a.out, a.ldo, a.out_f32 = out.data_ptr(), out.stride(0), int(out.dtype == F32)
        for k, v in kw.items():
            setattr(a, k, v.data_ptr() if isinstance(v, torch.Tensor) else v)
        K.gemv(a)
        return out.double()

    def near(got, ref):
        assert float((got - ref).abs().max()) < tol * float(ref.abs().max())

    W = w[:, :d].double()
    rms = lambda v: v / torch.sqrt((v * v).mean(-1, keepdim=True) + 1e-4)
    xn = x.double() + rms(y.double()) * w1.double()
    out, xo = torch.zeros(B, N, device="cuda"), torch.zeros(B, d, device="cuda")
    near(run(N, out, prologue=1, x=x, y=y, ldy=d, w1=w1, x_out=xo), xn @ W[:N].t())
    assert float((xo.double() - xn).abs().max()) < 1e-5
    near(run(N, out, prologue=1, x=x), x.double() @ W[:N].t())
    if d <= K.FINAL_NORM_MAX:
        near(run(N, out, prologue=1, x=x, y=y, ldy=d, w1=w1, w2=w2, softcap=3.0), 3.0 * torch.tanh(rms(xn) * w2.double() @ W[:N].t() / 3.0))
    act = torch.zeros(B, E, dtype=dtype, device="cuda")
    j = torch.arange(E)
    gate, up = W[(j // 64) * 128 + j % 64], W[(j // 64) * 128 + j % 64 + 64]
    gv = xn @ gate.t()
    near(run(2 * E, act, prologue=1, x=x, y=y, ldy=d, w1=w1, swiglu=1), gv * torch.sigmoid(gv) * (xn @ up.t()))
    x16 = torch.zeros(B, Kp, dtype=dtype, device="cuda")
    x16[:, :d] = x.to(dtype)
    near(run(N, out, prologue=0, x16=x16, ldx=Kp), x16[:, :d].double() @ W[:N].t())
    for parts in (1, 2, d // 2):
        if d % parts:
            continue
        z = torch.randn(B, d, generator=g).to(dtype).cuda()
        v = x16[:, :d].double() * z.double() * torch.sigmoid(z.double())
        v = rms(v.view(B, parts, -1)).reshape(B, d) * w1.double()
        if parts <= 256:
            gated = x16[:, :d].float() * (z.float() * torch.sigmoid(z.float()))
            sq = (gated * gated).view(B, parts, -1).sum(-1).contiguous()
            sq = torch.stack([sq * 0.25, sq * 0.75], -1).reshape(B, 2 * parts).contiguous()
            near(run(N, out, prologue=3, v32=gated, sq=sq, n_sq=2 * parts, w1=w1, parts=parts), v @ W[:N].t())
        near(run(N, out, prologue=2, y16=x16, ldy16=Kp, z16=z, ldz=d, w1=w1, parts=parts), v @ W[:N].t())


# ------------------------------------------------------------------------------------------------ long decoding, slots, batches
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_wrapping_rings(dtype):
    raw, w = C.edge_case()
    ids = C.tokens(raw, 700, 21)
    want = O.run(raw, C.as_numpy(w), ids)
    eng = engine(raw, w, dtype, max_len=2048, prefill_chunk=64)           # 128 ring rows: wraps five times
    assert eng.mem.layers[0].cap < 150 and eng.token_limit is None
    d = C.distance(feed(eng, "a", ids, [40] + list(range(41, 700))), want)
    assert d.max() < LIMIT[dtype], int(d.argmax())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(C.cases()))
def test_a_slot_used_again_remembers_nothing(name, dtype):
    raw, w, ids, want = case(name)
    fresh = feed(engine(raw, w, dtype), "b", ids[:80], [33, 34, 35])
    eng = engine(raw, w, dtype, batch=1)
    feed(eng, "a", C.tokens(raw, 200, 77), [64, 65])
    eng.end("a")
    assert np.array_equal(feed(eng, "b", ids[:80], [33, 34, 35]), fresh)


@pytest.mark.parametrize("dtype", DTYPES)
def test_open_requests_do_not_touch_each_other(dtype):
    raw, w, ids, _ = case("odd")
    other = C.tokens(raw, 300, 55)
    alone = [feed(engine(raw, w, dtype), "x", t[:90], [30, 31, 60]) for t in (ids, other)]
    eng = engine(raw, w, dtype, batch=3)
    out = {"p": [], "q": []}
    for lo, hi in ((0, 30), (30, 31), (31, 60), (60, 90)):
        for key, t in (("p", ids), ("q", other)):
            out[key].append(eng.step(key, t[lo:hi], range(hi - lo)).cpu().numpy())
    for key, ref in zip("pq", alone):
        assert np.array_equal(np.concatenate(out[key]), ref)
    eng.end("p")
    eng.end("q")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [1, 3, 9])
@pytest.mark.parametrize("name", sorted(C.cases()))
def test_batches_through_the_generator_interface(name, dtype, B):
    """Prompts of a batch and their token steps (GEMV chain, or GEMMs from eight sequences on) against each alone."""
    raw, w, _, _ = case(name)
    n, new = 33, 12
    seqs = [C.tokens(raw, n + new, 100 + b) for b in range(B)]
    wn = C.as_numpy(w)
    eng = engine(raw, w, dtype, batch=B, max_len=256)
    eng.reset(1)
    eng.prefill(torch.tensor([s[:n] for s in seqs], dtype=torch.int32))
    got = [[eng.logits[b].cpu().numpy()] for b in range(B)]
    for t in range(n, n + new - 1):
        eng.cur_tok.copy_(torch.tensor([s[t] for s in seqs], dtype=torch.int32))
        eng._forward_token()
        for b in range(B):
            got[b].append(eng.logits[b].cpu().numpy())
    eng.check()
    for b in range(0, B, 4):
        d = C.distance(np.stack(got[b]), O.run(raw, wn, seqs[b][:-1])[n - 1:])
        assert d.max() < LIMIT[dtype], (b, d.max())


# ------------------------------------------------------------------------------------------------ generation
def _greedy_oracle(raw, w, ids, new):
    ids, margins = list(ids), []
    for _ in range(new):
        lg = O.run(raw, w, ids)[-1]
        top = np.sort(lg)[-2:]
        margins.append(top[1] - top[0])
        ids.append(int(lg.argmax()))
    return ids[-new:], margins


@pytest.mark.parametrize("name", sorted(C.cases()))
def test_greedy_generation(name):
    from ghassan_b200.inference.generator import Generator
    from ghassan_b200.inference.token_loop import SamplingParams
    raw, w, ids, _ = case(name)
    want, margins = _greedy_oracle(raw, C.as_numpy(w), ids[:40], 24)
    sp = SamplingParams(greedy=True, repetition_penalty=1.0)
    assert min(margins) > 1e-3                               # no near-tie decides a token
    for use_graph in (True, False):
        gen = Generator(engine(raw, w, F32, max_len=256))
        res = gen.generate([ids[:40]], max_new_tokens=24, sampling=sp, stop_tokens=(), use_graph=use_graph)
        assert res.tokens[0] == want
    # the same engine again, and the captured step after another prompt
    assert gen.generate([ids[:40]], max_new_tokens=24, sampling=sp, stop_tokens=()).tokens[0] == want


@pytest.mark.parametrize("B", [1, 2, 8])
def test_bf16_generation_replays_its_steps(B):
    """The captured token step gives the tokens that single steps of the same engine give."""
    from ghassan_b200.inference.generator import Generator
    from ghassan_b200.inference.token_loop import SamplingParams
    raw, w, ids, _ = case("tiles")
    prompts = [C.tokens(raw, 50, 300 + b) for b in range(B)]
    sp = SamplingParams(greedy=True, repetition_penalty=1.0)
    a = Generator(engine(raw, w, BF, batch=B, max_len=256)).generate(prompts, max_new_tokens=40, sampling=sp, stop_tokens=())
    b = Generator(engine(raw, w, BF, batch=B, max_len=256)).generate(prompts, max_new_tokens=40, sampling=sp, stop_tokens=(), use_graph=False)
    assert a.tokens == b.tokens and all(len(t) == 40 for t in a.tokens)


def test_sampling_settings_and_stop_tokens_apply():
    from ghassan_b200.inference.generator import Generator
    from ghassan_b200.inference.token_loop import SamplingParams
    raw, w, ids, _ = case("odd")
    gen = Generator(engine(raw, w, BF, max_len=256))
    sp = SamplingParams(temperature=1.0, top_k=50, seed=7)
    one = gen.generate([ids[:20]], max_new_tokens=30, sampling=sp, stop_tokens=()).tokens[0]
    assert one == gen.generate([ids[:20]], max_new_tokens=30, sampling=sp, stop_tokens=()).tokens[0]
    assert one != gen.generate([ids[:20]], max_new_tokens=30, sampling=SamplingParams(temperature=1.0, top_k=50, seed=8), stop_tokens=()).tokens[0]
    cut = gen.generate([ids[:20]], max_new_tokens=30, sampling=sp, stop_tokens=(one[9],))
    assert cut.tokens[0] == one[:one.index(one[9])] and cut.stopped == ["eos"]
    host = gen.generate([ids[:20]], max_new_tokens=5, sampling=SamplingParams(greedy=True, no_repeat_ngram=2), stop_tokens=())
    assert len(host.tokens[0]) == 5
    nll, cnt = gen.score_tokens(ids[:30])
    want = O.run(raw, C.as_numpy(w), ids[:30])
    lp = want - np.log(np.exp(want).sum(-1, keepdims=True))
    assert cnt == 29 and abs(nll - -sum(lp[j, ids[j + 1]] for j in range(29))) < 0.02 * abs(nll)


def test_requests_that_cannot_be_served_are_refused():
    raw, w, ids, _ = case("odd")
    eng = engine(raw, w, BF, max_len=100, prefill_chunk=100)
    for bad in ([], [331], [-1]):
        with pytest.raises(ValueError):
            eng.step("a", bad)
    with pytest.raises(ValueError):
        eng.step("a", ids[:5], [5])
    assert eng.token_limit is not None
    with pytest.raises(ValueError, match="exceed"):
        eng.step("a", ids[:200])
    eng.end("a") if "a" in eng.mem.owner else None
    from ghassan_b200.inference.generator import Generator
    res = Generator(eng).generate([ids[:80]], max_new_tokens=100, stop_tokens=())
    assert len(res.tokens[0]) == eng.token_limit - 80 + 1


# ------------------------------------------------------------------------------------------------ command lines
def _model_folder(tmp_path, name):
    from test_layers_cpu import write_model
    return write_model(tmp_path / name, name)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run_program(tmp_path, dtype):
    raw, w, ids, want = case("odd")
    path, out = _model_folder(tmp_path, "odd"), tmp_path / "out"
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:70], "want": [0, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[70:71], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ids[71:73], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": ids[73:120], "want": [46]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": ids[:31], "want": [30]}], "end": ["b"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "120"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == ["done %d" % k for k in range(5)]
    got = np.concatenate([np.fromfile(out / ("%d.f32" % k), "<f4").reshape(-1, raw["vocab"]) for k in (0, 1, 3, 4)])
    d = C.distance(got, want[[0, 69, 70, 119, 30]])
    assert d.max() < LIMIT[BF if dtype == "bfloat16" else F32] * 2 and not (out / "2.f32").exists()


def test_inference_command_line(tmp_path, capsys):
    from ghassan_b200.cli import infer
    raw, w, ids, _ = case("odd")
    path = _model_folder(tmp_path, "odd")
    want, _ = _greedy_oracle(raw, C.as_numpy(w), ids[:12], 10)
    args = ["--model", path, "--ids", " ".join(map(str, ids[:12])), "--format", "f32"]
    assert infer.main(["generate", "--greedy", "--repeat", "1.0", "--max-tokens", "10"] + args) == 0
    assert capsys.readouterr().out.split() == [str(t) for t in want]
    assert infer.main(["logits", "--out", str(tmp_path / "l.f32")] + args) == 0
    lg = np.fromfile(tmp_path / "l.f32", "<f4")
    assert C.distance(lg[None], O.run(raw, C.as_numpy(w), ids[:12])[-1:]).max() < LIMIT[F32] * 2
    assert infer.main(["bench", "--model", path, "--tokens", "24", "--prompt-tokens", "20"]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["decode_tokens_per_s"] > 0
