"""Models with side-by-side sublayers on the device against the plain oracle: every mechanism alone, whole prompts, portions,
decoding, batches of unequal requests, slots that are used again, and generation through the framework's own entry points."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import dunavik_cases as D
import layers_cases as C
import layers_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

BF, F32 = torch.bfloat16, torch.float32
LIMIT = {BF: 0.06, F32: 2e-5}            # distance of logits; a planted mistake moves them by 0.2 and more
DTYPES = [F32, BF]
NAMES = sorted(D.cases())
_oracle = {}


def engine(raw, w, dtype, **kw):
    from ghassan_b200.inference.layer_engine import LayerEngine
    from ghassan_b200.models.layer_list import LayerListConfig
    return LayerEngine(LayerListConfig.from_json(raw), w, dtype=dtype, **kw)


def oracle(name, n=300, seed=0):
    raw = D.cases()[name]
    w, ids = D.weights(raw, seed), C.tokens(raw, n, seed + 11)
    key = (name, n, seed)
    if key not in _oracle:
        _oracle[key] = O.run(raw, C.as_numpy(w), ids, True)
    return raw, w, ids, _oracle[key]


def case(name, n=300, seed=0):
    raw, w, ids, (logits, _) = oracle(name, n, seed)
    return raw, w, ids, logits


def feed(eng, key, ids, cuts):
    """All logits of ``ids`` given in portions that end at ``cuts``."""
    out, lo = [], 0
    for hi in list(cuts) + [len(ids)]:
        if hi > lo:
            out.append(eng.step(key, ids[lo:hi], range(hi - lo)).cpu().numpy())
            lo = hi
    eng.check()
    return np.concatenate(out)


def near(got, want, tol):
    got, want = (np.asarray(t.double().cpu() if isinstance(t, torch.Tensor) else t, dtype=np.float64) for t in (got, want))
    assert np.abs(got - want).max() <= tol * np.abs(want).max(), np.abs(got - want).max() / np.abs(want).max()


# ------------------------------------------------------------------------------------------------ whole prompts and portions
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("cuts", [(), tuple(range(1, 300)), (2, 4, 7, 8, 129, 131, 299), tuple(range(2, 300, 2)), (40, 44, 49, 200), (128, 256),
                                  (17, 20, 34, 161)], ids=["whole", "tokens", "mixed", "pairs", "few", "tiles", "odd"])
def test_prompts_portions_and_tokens(name, dtype, cuts):
    raw, w, ids, want = case(name)
    d = C.distance(feed(engine(raw, w, dtype), "a", ids, cuts), want)
    assert d.max() < LIMIT[dtype], (d.max(), int(d.argmax()))


@pytest.mark.parametrize("name", NAMES)
def test_prompts_longer_than_a_pass_are_cut_inside(name):
    raw, w, ids, want = case(name)
    eng = engine(raw, w, F32, prefill_chunk=37, max_len=4000)
    assert C.distance(feed(eng, "a", ids, []), want).max() < LIMIT[F32]


@pytest.mark.parametrize("name", NAMES)
def test_tensor_core_kernels_and_general_kernels_agree(name):
    raw, w, ids, _ = case(name)
    a = feed(engine(raw, w, BF), "a", ids, [190])
    b = feed(engine(raw, w, BF, use_tensor_cores=False), "a", ids, [190])
    assert C.distance(a, b).max() < LIMIT[BF]


@pytest.mark.parametrize("name", NAMES)
def test_residual_after_every_run(name):
    raw, w, ids, (_, want) = oracle(name)
    eng = engine(raw, w, F32)
    s = eng.mem.acquire("a")
    seen = []
    eng._rows(torch.tensor(ids, dtype=torch.int32, device="cuda"), s, 1, len(ids), lambda i, x: seen.append(x.cpu().numpy()))
    assert len(seen) == len(want)
    for a, b in zip(seen, want):
        near(a, b, 1e-5)


# ------------------------------------------------------------------------------------------------ edges
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
@pytest.mark.parametrize("cuts", [(), tuple(range(1, 300)), (59, 60, 61, 95, 128, 131, 143, 257, 259), (5, 6, 96, 97, 112, 140, 176, 270),
                                  tuple(range(3, 300, 3)), (127,) + tuple(range(128, 300))], ids=["whole", "tokens", "a", "b", "threes", "tail"])
def test_window_edges_and_far_keys(dtype, kind, cuts):
    raw, w = D.edge_case(kind)
    ids, places = D.edge_tokens()
    if kind not in _oracle:
        _oracle[kind] = O.run(raw, C.as_numpy(w), ids)
    d = C.distance(feed(engine(raw, w, dtype), "a", ids, cuts), _oracle[kind])
    assert d.max() < LIMIT[dtype], {k: d[v].max() for k, v in places.items()}


@pytest.mark.parametrize("window, vdim, cap", [(128, 64, 20.0), (129, 128, 59.0), (300, 64, 8.0), (257, 128, 30.0), (1, 64, 20.0)])
def test_tensor_core_attention_at_tile_edges(window, vdim, cap):
    """Windows on and beside tile borders, long prompts cut at awkward places, a ring that wraps."""
    raw = D.config([D.attn(2, 1, 64, vdim, window, scale=0.12, cap=cap)], 64, 400, mult=1.0)
    w = D.weights(raw, 3, match=True)
    ids = C.tokens(raw, 900, 4, lo=200)
    rare = iter(range(0, 200, 2))
    for p in (450, 513, 641, 768, 895):
        for back in (window - 1, window):
            if 0 < back <= p and ids[p - back] >= 200 and ids[p] >= 200:
                t = next(rare)
                ids[p - back], ids[p] = t + 1, t
    want = O.run(raw, C.as_numpy(w), ids)
    for cuts in ((), (1, 300, 301, 640), (257, 512, 770)):
        d = C.distance(feed(engine(raw, w, BF, max_len=900, prefill_chunk=400), "a", ids, cuts), want)
        assert d.max() < LIMIT[BF], (cuts, d.max(), int(d.argmax()))
        assert C.distance(feed(engine(raw, w, F32, max_len=900, prefill_chunk=400), "a", ids, cuts), want).max() < LIMIT[F32]


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["rms", "layer"])
@pytest.mark.parametrize("rows, d", [(1, 33), (9, 84), (20, 1024), (3, 1028), (5, 4100), (2, 9001), (2, 12288)])
def test_embedding_and_residual_norms(dtype, kind, rows, d):
    from ghassan_b200.ops import layers as K
    g = torch.Generator().manual_seed(d)
    r = lambda *s: torch.randn(*s, generator=g).cuda()
    w, b = 1 + 0.2 * r(d), (0.3 * r(d) if kind == "layer" else None)
    ref = lambda v: (O.layer_norm(v, w.double().cpu().numpy(), b.double().cpu().numpy(), 1e-3) if kind == "layer"
                     else O.rms(v, 1e-3) * w.double().cpu().numpy())
    tol = 2e-6 if dtype == F32 else 2.0 ** -8
    n = lambda t: t.double().cpu().numpy()
    table = torch.zeros(17, (d + 7) // 8 * 8, device="cuda", dtype=dtype)
    table[:, :d] = (r(17, d) + 2.0).to(dtype)
    ids = torch.arange(rows, dtype=torch.int32, device="cuda") % 17
    x = torch.zeros(rows, d, device="cuda")
    K.embed_norm(ids, table, (kind, w, b), 1e-3, x, dtype)
    near(x, ref(n(table[ids.long(), :d])), 2e-6)
    y, x0 = r(rows, (d + 3) // 4 * 4), r(rows, d)
    x = r(rows, d) + 5.0
    for use_y, use_x0 in ((0, 0), (1, 0), (0, 1), (1, 1)):
        v = n(x) + (0.37 * n(y[:, :d]) if use_y else 0.0) + (n(x0) if use_x0 else 0.0)
        out = torch.full((rows, (d + 7) // 8 * 8), 9.0, dtype=dtype, device="cuda")
        for in_place in (False, True):
            xi = x.clone()
            xo = xi if in_place else torch.zeros_like(x)
            K.add_norm(xi, rows, (kind, w, b), 1e-3, out, y if use_y else None, 0.37, x0 if use_x0 else None, xo)
            near(xo, v, 1e-6)
            near(out[:, :d], ref(v), tol)
            assert float(out[:, d:].abs().sum()) == 0.0
        xo = torch.zeros_like(x)
        K.add_norm(x, rows, y=y if use_y else None, alpha=0.37, x0=x0 if use_x0 else None, x_out=xo)
        near(xo, v, 1e-6)
    pick = torch.tensor([rows - 1, 0, rows // 2], dtype=torch.int32, device="cuda")
    out = torch.zeros(3, (d + 7) // 8 * 8, dtype=dtype, device="cuda")
    K.add_norm(x, 3, (kind, w, b), 1e-3, out, row_idx=pick)
    near(out[:, :d], ref(n(x)[pick.cpu().numpy()]), tol)


@pytest.mark.parametrize("M, N, Kd, pair", [(5, 40, 72, False), (300, 136, 200, False), (130, 256, 64, False), (512, 512, 136, True), (700, 600, 96, True)])
def test_product_with_squared_positive_part(M, N, Kd, pair):
    from ghassan_b200.ops import _lib
    from ghassan_b200.ops import gemm as G
    g = torch.Generator().manual_seed(M)
    a, b = (torch.randn(M, Kd, generator=g).to(BF).cuda(), (torch.randn(N, Kd, generator=g) * Kd ** -0.5).to(BF).cuda())
    wide = torch.full((M, N + 24), 7.0, dtype=BF, device="cuda")
    G.gemm(a, b, out=wide[:, 16:16 + N], relu2=True, pair=pair)
    _lib.check_status(a.device)
    near(wide[:, 16:16 + N], torch.relu(a.double() @ b.double().t()) ** 2, 2.0 ** -8)
    assert bool((wide[:, :16] == 7.0).all()) and bool((wide[:, 16 + N:] == 7.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [1, 3, 8])
@pytest.mark.parametrize("d, N, n1", [(36, 50, 13), (300, 333, 290), (2100, 70, 0), (5000, 24, 8)])
def test_gemv_prologues(dtype, B, d, N, n1):
    """Residual add with the norm ahead, the norm of a latent, rows that leave as squared positive parts."""
    from ghassan_b200.ops import layers as K
    g = torch.Generator().manual_seed(d + N)
    Kp = (d + 7) // 8 * 8
    w = torch.zeros(N, Kp, dtype=dtype, device="cuda")
    w[:, :d] = (torch.randn(N, d, generator=g) * d ** -0.5).to(dtype).cuda()
    x, y, x0 = (torch.randn(B, d, generator=g).cuda() for _ in range(3))
    w1, b1 = 1 + 0.1 * torch.randn(d, generator=g).cuda(), 0.2 * torch.randn(d, generator=g).cuda()
    tol = 1e-5 if dtype == F32 else 2.0 ** -6
    W = w[:, :d].double()
    for mode in ("rms", "layer"):
        for use_y, use_x0, bias in ((1, 1, 1), (1, 0, 0), (0, 1, 1), (0, 0, 1)):
            a = K.GemvArgs()
            a.W, a.fmt, a.N, a.K, a.B, a.dtype, a.d, a.eps, a.prologue, a.norm_mode = w.data_ptr(), K.W_FMT[dtype], N, Kp, B, K.DTYPE[dtype], d, 1e-4, 5, K.NORM[mode]
            out, xo = torch.zeros(B, N, device="cuda"), torch.zeros(B, d, device="cuda")
            out2 = torch.zeros(B, N, dtype=dtype, device="cuda")
            a.out, a.ldo, a.out_f32, a.x, a.w1, a.x_out, a.alpha = out.data_ptr(), N, 1, x.data_ptr(), w1.data_ptr(), xo.data_ptr(), 0.7
            a.n1, a.out2, a.ldo2 = n1, out2.data_ptr(), N
            if use_y:
                a.y, a.ldy = y.data_ptr(), d
            if use_x0:
                a.x0 = x0.data_ptr()
            if bias:
                a.b1 = b1.data_ptr()
            K.gemv(a)
            v = x.double() + 0.7 * use_y * y.double() + use_x0 * x0.double()
            near(xo, v, 1e-6)
            c = v - v.mean(-1, keepdim=True) if mode == "layer" else v
            h = c / torch.sqrt((c * c).mean(-1, keepdim=True) + 1e-4) * w1.double() + bias * b1.double()
            ref = h @ W.t()
            k = n1 or N
            near(out[:, :k], ref[:, :k], tol)
            if n1:
                near(out2[:, :N - n1], torch.relu(ref[:, n1:]) ** 2, 4 * tol)
                assert float(out[:, n1:].abs().sum()) == 0.0
    v16 = torch.zeros(B, Kp + 8, dtype=dtype, device="cuda")
    v16[:, :d] = x.to(dtype)
    a = K.GemvArgs()
    a.W, a.fmt, a.N, a.K, a.B, a.dtype, a.d, a.eps, a.prologue = w.data_ptr(), K.W_FMT[dtype], N, Kp, B, K.DTYPE[dtype], d, 1e-4, 4
    out = torch.zeros(B, N, device="cuda")
    a.out, a.ldo, a.out_f32, a.x16, a.ldx, a.w1 = out.data_ptr(), N, 1, v16.data_ptr(), Kp + 8, w1.data_ptr()
    K.gemv(a)
    v = v16[:, :d].double()
    near(out, (v / torch.sqrt((v * v).mean(-1, keepdim=True) + 1e-4) * w1.double()) @ W.t(), tol)


def _one_layer(layer, width=64, dtype=F32, slots=1, rows=512, max_len=4096, seed=0, tc=True):
    """A model of one layer and its memory, for kernels on hand-made projections."""
    from ghassan_b200.inference.layer_cache import SlotManager
    from ghassan_b200.models.layer_list import LayerListConfig
    from ghassan_b200.models.layer_model import LayerModel
    raw = D.config([layer], width, 32)
    cfg = LayerListConfig.from_json(raw)
    m = LayerModel(cfg, D.weights(raw, seed), slots, rows, dtype, use_tensor_cores=tc)
    mem = SlotManager(cfg, slots, max_len, rows, dtype, m.dev)
    return m, mem, torch.zeros(slots, 4, dtype=torch.int32, device="cuda")


def _projection(m, rows, seed=3):
    src = m.buf("proj", (m.weights[0].w_in.shape[0] + 7) // 8 * 8)
    src[:rows] = torch.randn(rows, src.shape[1], generator=torch.Generator().manual_seed(seed)).to(m.dtype).cuda()
    return src[:rows].double().cpu().numpy()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim, every, coef, pos", [(24, 1, 1.0, 0), (64, 7, 0.5, 1000), (20, 100, -0.2, 199), (256, 65536, 0.9, 131070)])
def test_query_temperature(dtype, dim, every, coef, pos):
    """Positions on both sides of a step of the factor; keys and values stay as they are."""
    from ghassan_b200.ops import layers as K
    m, mem, state = _one_layer(D.attn(3, 1, dim, 16, 50, coef=coef, every=every), dtype=dtype)
    n = 6
    proj = _projection(m, n)
    state[:, 0] = pos
    a = m.attn_args(0, mem.layers[0], state, 0, 1, n, -1)
    K.qkv_store(a)
    p = np.arange(pos, pos + n)
    q = proj[:, :3 * dim].reshape(n, 3, dim) * O.query_temperature(p, coef, every)[:, None, None]
    near(m.buf("q", 3 * a.dkp)[:n].view(n, 3, a.dkp)[..., :dim], q, 1e-6 if dtype == F32 else 2.0 ** -8)
    c = mem.layers[0]
    rows = [int(x) % c.cap for x in p]
    near(c.k[0, rows, 0, :dim], proj[:, 3 * dim:4 * dim], 0.0)
    near(c.v[0, rows, 0, :16], proj[:, 4 * dim:4 * dim + 16], 0.0)


def _attention_oracle(proj, mx, positions):
    """Soft-max attention of the plain equations on hand-made projections of one sequence."""
    T, H, G, dk, dv = len(positions), mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = proj[:, :H * dk].reshape(T, H, dk) * O.query_temperature(positions, mx["q_temp"]["coef"], mx["q_temp"]["every"])[:, None, None]
    k = proj[:, H * dk:(H + G) * dk].reshape(T, G, dk)
    v = proj[:, (H + G) * dk:(H + G) * dk + G * dv].reshape(T, G, dv)
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    see = (back >= 0) & (back < mx["mask"]["size"])
    out = np.zeros((T, H, dv))
    for h in range(H):
        g = h // (H // G)
        s = O.soft_cap(q[:, h] @ k[:, g].T * mx["scale"], mx["softcap"]) - O.distance_slopes(H)[h] * back
        out[:, h] = O.softmax(s, see) @ v[:, g]
    return out.reshape(T, H * dv)


@pytest.mark.parametrize("H, G, dim, vdim, window, cap", [(4, 2, 64, 64, 100, 15.0), (6, 6, 40, 128, 128, 50.0), (8, 1, 128, 96, 300, 2.0), (1, 1, 96, 48, 257, 30.0),
                                                          (3, 1, 160, 200, 90, 70.0)])
@pytest.mark.parametrize("kernel", ["tc", "general", "general fp32", "tokens", "tokens fp32"])
def test_capped_and_biased_attention(H, G, dim, vdim, window, cap, kernel):
    from ghassan_b200.ops import _lib
    from ghassan_b200.ops import layers as K
    layer = D.attn(H, G, dim, vdim, window, scale=0.5, cap=cap, coef=0.1, every=50)
    dtype = F32 if kernel.endswith("fp32") else BF
    T = 330
    m, mem, state = _one_layer(layer, dtype=dtype)
    proj = _projection(m, T)
    want = _attention_oracle(proj, layer["mixer"], range(T))
    out = m.mixed(0)
    if kernel.startswith("tokens"):
        src, got = m.buf("proj", (m.weights[0].w_in.shape[0] + 7) // 8 * 8), []
        whole = src[:T].clone()
        for t in range(T):
            src[:1] = whole[t:t + 1]
            a = m.attn_args(0, mem.layers[0], state, 0, 1, 1, -1)
            K.qkv_store(a)
            K.attn_decode(a)
            got.append(out[:1, :H * vdim].clone())
            state[:, 0] += 1
        got = torch.cat(got)
    else:
        a = m.attn_args(0, mem.layers[0], state, 0, 1, T, 0)
        K.qkv_store(a)
        if kernel == "tc":
            if cap > 60 or dim > 128:
                assert not K.attn_tc_ok(a)
                return
            assert K.attn_tc_ok(a)
        (K.attn_tc if kernel == "tc" else K.attn_prefill)(a)
        got = out[:T, :H * vdim]
    _lib.check_status(m.dev)
    near(got, want, 1e-5 if dtype == F32 else 2.0 ** -6)


LATENTS = [(3, 20, 10, 28, 44, 36), (6, 64, 32, 64, 96, 40), (1, 128, 64, 128, 256, 200), (5, 16, 64, 24, 512, 64), (2, 30, 34, 20, 700, 1040), (9, 8, 8, 8, 8, 8)]


def _latent_reference(m, proj, positions, dtype):
    """Latent rows, queries and gated outputs of the plain equations on a hand-made projection; the pieces that the device keeps
    in its compute type are rounded as it does."""
    mx, w = m.cfg.layers[0].mixer, C.as_numpy(D.weights(D.config([_raw_of(m)], 64, 32)))
    rnd = lambda t: torch.from_numpy(np.asarray(t)).to(dtype).double().numpy()
    T, H, dn, dr, dv, R, Q = len(positions), mx.heads, mx.dim, mx.rot_dim, mx.vdim, mx.kv_rank, mx.q_rank
    rot = {"base": mx.rot.base, "dims": mx.rot.dims}
    w = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    cq = rnd(O.rms(proj[:, :Q], m.cfg.eps) * w["l0.mix.dq.norm"])
    c = rnd(O.rms(proj[:, Q:Q + R], m.cfg.eps) * w["l0.mix.dkv.norm"])
    kr = rnd(O.rotate(proj[:, None, Q + R:Q + R + dr], rot, positions)[:, 0])
    q = rnd(cq @ w["l0.mix.uq"].T).reshape(T, H, dn + dr)
    q[..., dn:] = O.rotate(q[..., dn:], rot, positions)
    k = np.concatenate([(c @ w["l0.mix.uk"].T).reshape(T, H, dn), np.repeat(kr[:, None], H, 1)], -1)
    v = (c @ w["l0.mix.uv"].T).reshape(T, H, dv)
    see = np.tril(np.ones((T, T), dtype=bool))
    out = np.stack([O.softmax(q[:, h] @ k[:, h].T * mx.scale, see) @ v[:, h] for h in range(H)], 1).reshape(T, H * dv)
    return np.concatenate([c, kr], -1), cq, q, out * O.sigmoid(proj[:, Q + R + dr:Q + R + dr + H * dv])


def _raw_of(m):
    x = m.cfg.layers[0].mixer
    return D.latent(x.heads, x.dim, x.rot_dim, x.vdim, x.kv_rank, x.q_rank, base=x.rot.base)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", LATENTS, ids=["x".join(map(str, s)) for s in LATENTS])
@pytest.mark.parametrize("pos", [0, 1000])
def test_latent_rows_and_queries(dtype, sizes, pos):
    from ghassan_b200.ops import layers as K
    m, mem, state = _one_layer(D.latent(*sizes), dtype=dtype)
    n, w = 9, m.weights[0]
    proj = _projection(m, n)
    state[:, 0] = pos
    rows, cq, q, _ = _latent_reference(m, proj, range(pos, pos + n), dtype)
    m._rotations(state, 1, n)
    a = m.latent_args(0, mem.layers[0], state, 0, 1, n)
    K.latent_store(a)
    tol = 3e-6 if dtype == F32 else 2.0 ** -7
    D_ = rows.shape[1]
    near(mem.layers[0].rows[0, pos:pos + n, :D_], rows, tol)
    assert float(mem.layers[0].rows[0, :, D_:].abs().sum()) == 0.0 and float(mem.layers[0].rows[0, pos + n:].abs().sum()) == 0.0
    near(m.buf("cq", w.w_uq.shape[1])[:n, :sizes[5]], cq, tol)
    m._gemm(m.buf("cq", w.w_uq.shape[1]), w.w_uq, m.buf("qc", (w.w_uq.shape[0] + 7) // 8 * 8), n)
    K.latent_queries(a)
    got = m.buf("q", sizes[0] * a.dkp)[:n].view(n, sizes[0], a.dkp)
    near(got[..., :sizes[1] + sizes[2]], q, 4 * tol)
    assert float(got[..., sizes[1] + sizes[2]:].abs().sum()) == 0.0


@pytest.mark.parametrize("dtype, tc", [(F32, False), (BF, False), (BF, True)], ids=["fp32", "general", "tc"])
@pytest.mark.parametrize("sizes", LATENTS, ids=["x".join(map(str, s)) for s in LATENTS])
@pytest.mark.parametrize("portions", [(200,), (1,) * 70, (130, 1, 2, 3, 4, 1, 59), (2, 5, 4, 140, 3), (505, 1, 1, 1, 3)],
                         ids=["whole", "tokens", "mixed", "few", "long"])
def test_latent_attention_of_portions(dtype, tc, sizes, portions):
    """Keys and values made for a pass, and queries against the latents themselves, over one cache."""
    from ghassan_b200.ops import _lib
    from ghassan_b200.ops import layers as K
    m, mem, state = _one_layer(D.latent(*sizes), dtype=dtype, tc=tc)
    T, w = sum(portions), m.weights[0]
    proj = _projection(m, T)
    want = _latent_reference(m, proj, range(T), dtype)[3]
    src, got, lo = m.buf("proj", (w.w_in.shape[0] + 7) // 8 * 8), [], 0
    whole = src[:T].clone()
    for n in portions:
        m.x16.zero_()
        src[:n] = whole[lo:lo + n]
        m._rotations(state, 1, n)
        gemm = m._gemm
        m._gemm = lambda a, b, out, rows: None if b is w.w_in else gemm(a, b, out, rows)      # the projection is given
        m._mix_rows(0, mem.layers[0], state, 0, 1, n, lo)
        m._gemm = gemm
        got.append(m.mixed(0)[:n, :sizes[0] * sizes[3]].clone())
        state[:, 0] += n
        lo += n
    _lib.check_status(m.dev)
    near(torch.cat(got), want, 2e-5 if dtype == F32 else 2.0 ** -5)


@pytest.mark.parametrize("H, rank, dr", [(5, 96, 32), (16, 256, 64), (20, 512, 64), (40, 64, 16), (33, 640, 64)])
@pytest.mark.parametrize("splits", [1, 2, 5])
def test_latent_tensor_core_partials(H, rank, dr, splits):
    """Runs of several tiles with a growing maximum, one key far above the others, against the plain soft-max; rows of the cache
    past the sequence hold other numbers."""
    from ghassan_b200.ops import _lib
    from ghassan_b200.ops import layers as K
    m, mem, state = _one_layer(D.latent(H, 16, dr, 24, rank, 32), dtype=BF, max_len=1500)
    g = torch.Generator().manual_seed(H)
    count = 1203
    c = mem.layers[0]
    c.rows[0, :, :rank + dr] = torch.randn(c.cap, rank + dr, generator=g).to(BF).cuda()
    c.rows[0, :count] *= torch.linspace(0.3, 1.0, count, device="cuda").to(BF)[:, None]
    state[:, 0] = count - 1
    m._rotations(state, 1, 1)
    a = m.latent_args(0, c, state, 0, 1, 1)
    a.scale, a.splits = 0.1, splits
    scratch = torch.zeros(H * splits * (a.ldc + 2), device="cuda")
    a.scratch = scratch.data_ptr()
    qa = torch.zeros(a.heads_pad, a.ld_qa16, dtype=BF, device="cuda")
    qa[:H, :rank + dr] = torch.randn(H, rank + dr, generator=g).to(BF).cuda() * (10.0 * (rank + dr) ** -0.5)
    qa[1, :rank + dr] = c.rows[0, 131, :rank + dr] * 0.6
    a.qa16 = qa.data_ptr()
    gate = torch.full((1, H * 24), 50.0, dtype=BF, device="cuda")
    a.gate, a.ld_gate = gate.data_ptr(), H * 24
    K.latent_attn(a)
    _lib.check_status(m.dev)
    rows = c.rows[0, :count, :rank + dr].double().cpu().numpy()
    s = qa[:H, :rank + dr].double().cpu().numpy() @ rows.T * 0.1
    o = O.softmax(s, np.ones_like(s, dtype=bool)) @ rows[:, :rank]
    values = m.weights[0].w_kv[H * a.dkp:].view(H, a.dvp, -1)[:, :24, :rank].double().cpu().numpy()
    near(m.mixed(0)[:1, :H * 24].view(H, 24), np.einsum("hvr,hr->hv", values, o), 2.0 ** -6)


# ------------------------------------------------------------------------------------------------ long decoding, slots, batches
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_wrapping_rings(dtype):
    raw, w = D.edge_case("attention")
    ids = C.tokens(raw, 700, 21)
    want = O.run(raw, C.as_numpy(w), ids)
    eng = engine(raw, w, dtype, max_len=1024, prefill_chunk=64)           # 128 ring rows: wraps five times
    assert eng.mem.layers[0].cap == 128 and eng.token_limit == 1024
    d = C.distance(feed(eng, "a", ids, [40] + list(range(41, 700))), want)
    assert d.max() < LIMIT[dtype], int(d.argmax())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_a_slot_used_again_remembers_nothing(name, dtype):
    raw, w, ids, want = case(name)
    fresh = feed(engine(raw, w, dtype), "b", ids[:80], [33, 34, 35, 38])
    eng = engine(raw, w, dtype, batch=1)
    feed(eng, "a", C.tokens(raw, 200, 77), [64, 65])
    eng.end("a")
    assert np.array_equal(feed(eng, "b", ids[:80], [33, 34, 35, 38]), fresh)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_open_requests_do_not_touch_each_other(name, dtype):
    raw, w, ids, _ = case(name)
    other = C.tokens(raw, 300, 55)
    cuts = (30, 31, 33, 60)
    alone = [feed(engine(raw, w, dtype), "x", t[:90], cuts) for t in (ids, other)]
    eng = engine(raw, w, dtype, batch=3)
    out, lo = {"p": [], "q": []}, 0
    for hi in cuts + (90,):
        for key, t in (("p", ids), ("q", other)):
            out[key].append(eng.step(key, t[lo:hi], range(hi - lo)).cpu().numpy())
        lo = hi
    for key, ref in zip("pq", alone):
        assert np.array_equal(np.concatenate(out[key]), ref)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [2, 8, 9])
@pytest.mark.parametrize("name", NAMES)
def test_token_steps_of_unequal_requests(name, dtype, B):
    """Requests of different lengths advance together (GEMV chain, or GEMMs from eight on), each as if it were alone."""
    raw, w, _, _ = case(name)
    lens = [3 + 29 * b for b in range(B)]
    seqs = [C.tokens(raw, n + 6, 100 + b) for b, n in enumerate(lens)]
    eng = engine(raw, w, dtype, batch=B, max_len=300)
    slots = []
    for b, n in enumerate(lens):
        eng.step(b, seqs[b][:n])
        slots.append(eng.mem.owner[b])
    got = [[] for _ in range(B)]
    for t in range(6):
        cur = [0] * B
        for b, s in enumerate(slots):
            cur[s] = seqs[b][lens[b] + t]
        eng.cur_tok.copy_(torch.tensor(cur, dtype=torch.int32))
        eng._forward_token()
        for b, s in enumerate(slots):
            got[b].append(eng.logits[s].cpu().numpy())
    eng.check()
    for b in range(0, B, 3):
        d = C.distance(np.stack(got[b]), O.run(raw, C.as_numpy(w), seqs[b])[lens[b]:])
        assert d.max() < LIMIT[dtype], (b, d.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [1, 3, 9])
@pytest.mark.parametrize("name", NAMES)
def test_batches_through_the_generator_interface(name, dtype, B):
    """Prompts of a batch, in one pass or several, and their token steps against each alone."""
    raw, w, _, _ = case(name)
    n, new = 33, 8
    seqs = [C.tokens(raw, n + new, 100 + b) for b in range(B)]
    eng = engine(raw, w, dtype, batch=B, max_len=256 if B < 9 else 600, prefill_chunk=20 if B == 3 else 2048)
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
        d = C.distance(np.stack(got[b]), O.run(raw, C.as_numpy(w), seqs[b][:-1])[n - 1:])
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


@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation(name):
    from ghassan_b200.inference.generator import Generator
    from ghassan_b200.inference.token_loop import SamplingParams
    raw, w, ids, _ = case(name)
    want, margins = _greedy_oracle(raw, C.as_numpy(w), ids[:40], 20)
    sp = SamplingParams(greedy=True, repetition_penalty=1.0)
    assert min(margins) > 1e-3                               # no near-tie decides a token
    for use_graph in (True, False):
        gen = Generator(engine(raw, w, F32, max_len=256))
        assert gen.generate([ids[:40]], max_new_tokens=20, sampling=sp, stop_tokens=(), use_graph=use_graph).tokens[0] == want
    # the same engine again, and the captured step after another prompt
    gen.generate([ids[50:77]], max_new_tokens=9, sampling=sp, stop_tokens=())
    assert gen.generate([ids[:40]], max_new_tokens=20, sampling=sp, stop_tokens=()).tokens[0] == want


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


def test_sequences_that_do_not_fit_are_refused():
    raw, w, ids, _ = case("odd")
    eng = engine(raw, w, BF, max_len=100)
    assert eng.token_limit == 128
    with pytest.raises(ValueError, match="exceed"):
        eng.step("a", ids[:200])


# ------------------------------------------------------------------------------------------------ command lines
def _model_folder(tmp_path, name):
    from ghassan_b200.formats import safetensors as ST
    raw = D.cases()[name]
    folder = tmp_path / name
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(raw))
    ST.save(str(folder / "model.safetensors"), D.weights(raw))
    return str(folder)


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
    assert infer.main(["bench", "--model", path, "--tokens", "24", "--prompt-tokens", "20"]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["decode_tokens_per_s"] > 0
