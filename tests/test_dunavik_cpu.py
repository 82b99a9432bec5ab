"""Models with side-by-side sublayers without a device: configuration, order of runs, memory of a sequence, and the power of the
inputs the GPU tests use (a mistake planted in the oracle shows in the logits)."""
import copy
import json

import numpy as np
import pytest
import torch

import dunavik_cases as D
import layers_cases as C
import layers_oracle as O
from ghassan_b200.models import registry
from ghassan_b200.models.layer_list import (AttentionMixer, LatentAttentionMixer, LayerListConfig, QueryTemperature, Rotary, Run, check_tensors,
                                            layer_runs, random_parameters)


@pytest.mark.parametrize("name", sorted(D.cases()))
def test_configuration_names_every_tensor(name):
    raw = D.cases()[name]
    cfg = registry.from_json(raw).parse(raw)
    w = D.weights(raw)
    assert {k: tuple(v.shape) for k, v in w.items()} == cfg.tensor_shapes()
    check_tensors(cfg, w)
    assert {k: tuple(v.shape) for k, v in random_parameters(cfg).items()} == cfg.tensor_shapes()
    assert [(r.layer, r.rejoin) for r in cfg.runs] == O.layer_runs(raw)
    assert registry.engine_class(cfg).__name__ == "LayerEngine"


def test_configuration_reads_every_field():
    raw = D.cases()["odd"]
    cfg = LayerListConfig.from_json(json.loads(json.dumps(raw)))
    a, b = cfg.layers[0].mixer, cfg.layers[1].mixer
    assert isinstance(a, AttentionMixer) and (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first) == (6, 2, 24, 40, 37, 0)
    assert (a.softcap, a.q_temp, a.distance_bias, a.rot) == (12.0, QueryTemperature(2.0, 5), True, None)
    assert not (a.qk_norm or a.sink or a.gate)
    np.testing.assert_allclose(a.slopes(), O.distance_slopes(6), rtol=1e-12)
    assert isinstance(b, LatentAttentionMixer) and (b.heads, b.dim, b.rot_dim, b.vdim, b.kv_rank, b.q_rank) == (3, 20, 10, 28, 44, 36)
    assert b.rot == Rotary(10, 10000.0) and b.scale == 30 ** -0.5
    assert (cfg.eps, cfg.residual_mult, cfg.logit_softcap, cfg.hidden_size, cfg.vocab_size) == (1e-5, 0.3, 0.0, 84, 331)
    assert cfg.layers[0].mlp.ff == 88 and cfg.layers[0].mlp.activation == "relu2" and cfg.layers[2].mlp is None


@pytest.mark.parametrize("loop, want", [(None, [0, 1, 2, 3]), ({"start": 0, "stop": 4, "times": 1}, [0, 1, 2, 3]),
                                        ({"start": 1, "stop": 3, "times": 3}, [0, 1, 2, -1, 2, -1, 2, 3]),
                                        ({"start": 3, "stop": 4, "times": 2}, [0, 1, 2, 3, -3])])
def test_order_of_runs(loop, want):
    assert layer_runs(4, loop) == [Run(abs(i), i < 0) for i in want]


@pytest.mark.parametrize("change, word", [
    (lambda d: d["layers"][0].update(type="mamba2"), "unknown layer type"),
    (lambda d: d["layers"][0]["mixer"].update(softcap=0), "softcap"),
    (lambda d: d["layers"][0]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda d: d["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda d: d["layers"][1]["mixer"].update(q_rank=0), "q_rank"),
    (lambda d: d["layers"][1]["mixer"].update(dim=250), "exceed"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=12), "exceeds"),
    (lambda d: d["loop"].update(stop=5), "stop"),
    (lambda d: d["loop"].update(start=3), "behind"),
    (lambda d: d["loop"].update(times=0), "times"),
    (lambda d: d.update(residual_mult="1"), "residual_mult"),
])
def test_configuration_mistakes_are_named(change, word):
    raw = copy.deepcopy(D.cases()["odd"])
    change(raw)
    with pytest.raises(ValueError, match=word):
        LayerListConfig.from_json(raw)


def test_other_designs_take_no_loop():
    with pytest.raises(ValueError, match="loop"):
        LayerListConfig.from_json(dict(C.cases()["odd"], loop={"start": 0, "stop": 1, "times": 2}))


def test_missing_biases_are_named():
    raw = D.cases()["odd"]
    cfg, w = LayerListConfig.from_json(raw), D.weights(raw)
    for n in ("embed.norm.b", "l2.norm1.b", "final.norm.b", "l1.mix.dkv.norm"):
        with pytest.raises(ValueError, match=n):
            check_tensors(cfg, {k: v for k, v in w.items() if k != n})


def test_every_run_has_a_memory_of_its_own():
    from ghassan_b200.inference.layer_cache import AttentionCache, LatentCache, SlotManager
    cfg = LayerListConfig.from_json(D.cases()["odd"])
    m = SlotManager(cfg, 2, 300, 16, torch.float32, "cpu")
    assert [type(c) for c in m.layers] == [AttentionCache] + [LatentCache, AttentionCache] * 3 + [LatentCache]
    kept = [c.rows.data_ptr() if isinstance(c, LatentCache) else c.k.data_ptr() for c in m.layers]
    assert len(set(kept)) == 8
    assert m.layers[1].rows.shape == (2, 384, 56) and m.limit == 384        # 44 + 10 numbers per token, padded
    with pytest.raises(ValueError, match="exceed"):
        m.claim(0, 1, 385)
    windows = SlotManager(LayerListConfig.from_json(dict(D.cases()["odd"], layers=[D.attn(2, 1, 8, 8, 5)], loop=None)), 1, 4096, 64, torch.float32, "cpu")
    assert windows.limit is None and windows.layers[0].cap == 128


# ------------------------------------------------------------------------------------------------ the oracle
def test_oracle_does_not_look_ahead():
    raw = D.cases()["odd"]
    w, ids = C.as_numpy(D.weights(raw, 3)), C.tokens(raw, 50)
    full = O.run(raw, w, ids)
    for n in (1, 7, 38):
        np.testing.assert_allclose(O.run(raw, w, ids[:n]), full[:n], atol=1e-9)


def _patched(name, f):
    def change(raw, w, mp):
        mp.setattr(O, name, f(getattr(O, name)))
    return change


def _edit(f):
    return lambda raw, w, mp: f(raw, w)


def _mixer(kind, **kw):
    def f(raw, w):
        for e in raw["layers"]:
            if e["type"] == kind:
                e["mixer"].update(kw)
    return _edit(f)


def _mutants():
    """kind -> (which model, mistake)."""
    window = lambda n: _mixer("attention", mask={"size": D.EDGE_WINDOW + n})
    return {
        "window_in": ("attention", window(-1)),
        "window_out": ("attention", window(1)),
        "far": ("latent_attention", _patched("latent_attention", lambda f: lambda h, mix, w, eps: np.concatenate(
            [f(h[max(0, t - 127):t + 1], mix, w, eps)[-1:] for t in range(len(h))]))),
        "cap": ("attention", _mixer("attention", softcap=1e6)),
        "slopes": ("attention", _patched("distance_slopes", lambda f: lambda heads: f(heads) * 2.0 ** (8.0 / heads))),
        "temperature": ("temper", _patched("query_temperature", lambda f: lambda p, c, e: np.ones(len(p)))),
        "temperature a token late": ("temper", _patched("query_temperature", lambda f: lambda p, c, e: f([max(x - 1, 0) for x in p], c, e))),
        "rotation": ("odd", _patched("rotate", lambda f: lambda x, rot, p: x)),
        "latent norm": ("odd", _patched("rms", lambda f: lambda x, eps: x)),
        "gate": ("odd", _edit(lambda raw, w: w.update({"l1.mix.g": w["l1.mix.g"] * 0}))),
        "rejoin": ("attention", _patched("layer_runs", lambda f: lambda cfg: [(i, False) for i, _ in f(cfg)])),
        "one run": ("attention", _edit(lambda raw, w: raw.update(loop=None))),
        "relu": ("attention", _patched("squared_relu_mlp", lambda f: lambda h, w: np.maximum(h @ w["up"].T, 0.0) @ w["down"].T)),
        "multiplier": ("attention", _edit(lambda raw, w: raw.update(residual_mult=0.5))),
    }


@pytest.mark.parametrize("kind", sorted(_mutants()))
def test_inputs_show_a_planted_mistake(kind, monkeypatch):
    """Each mistake moves the logits at its own places by far more than the GPU tests allow there."""
    model, change = _mutants()[kind]
    if model in D.cases():
        raw, places = D.cases()[model], {}
        w, ids = D.weights(raw), C.tokens(raw, 100)
    else:
        raw, w = D.edge_case(model)
        ids, places = D.edge_tokens()
    w = C.as_numpy(w)
    good = O.run(raw, w, ids)
    raw2, w2 = copy.deepcopy(raw), dict(w)
    change(raw2, w2, monkeypatch)
    d = C.distance(O.run(raw2, w2, ids), good)
    at = places.get(kind, [])
    assert (d[at].min() if at else d.max()) > 0.2, d[at] if at else d.max()


@pytest.mark.parametrize("change", ["centre", "bias", "embed"])
def test_norms_matter_in_the_general_cases(change, monkeypatch):
    raw = D.cases()["odd"]
    w, ids = C.as_numpy(D.weights(raw)), C.tokens(raw, 60)
    good = O.run(raw, w, ids)
    w2 = dict(w)
    if change == "centre":
        monkeypatch.setattr(O, "layer_norm", lambda x, g, b, eps: O.rms(x, eps) * g + b)
    elif change == "bias":
        w2.update({k: v * 0 for k, v in w.items() if k.endswith("norm1.b")})
    else:
        w2.update({"embed.norm": np.ones_like(w["embed.norm"])})
    assert C.distance(O.run(raw, w2, ids), good).max() > 0.2


def test_model_folder_loads(tmp_path, capsys):
    from ghassan_b200.cli import infer
    from ghassan_b200.formats import safetensors as ST
    from ghassan_b200.inference import model_io as IO
    raw = D.cases()["odd"]
    (tmp_path / "config.json").write_text(json.dumps(raw))
    ST.save(str(tmp_path / "model.safetensors"), D.weights(raw))
    m = IO.load_model(str(tmp_path))
    assert isinstance(m.cfg, LayerListConfig) and torch.equal(m.named["l1.mix.uk"], D.weights(raw)["l1.mix.uk"])
    assert infer.main(["info", "--model", str(tmp_path)]) == 0
    out = capsys.readouterr().out
    assert "Dunavik" in out and "latent_attention" in out
