"""Layer-list models without a device: configuration, files, rotation frequencies, sequence slots, the trace replay's
protocol, and the power of the inputs the GPU tests use (a mistake planted in the oracle shows in the logits)."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import layers_cases as C
import layers_oracle as O
from ghassan_b200.models import registry
from ghassan_b200.models.layer_list import AttentionMixer, LayerListConfig, Mamba2Mixer, Rotary, RotaryScaling, check_tensors, random_parameters


@pytest.mark.parametrize("name", sorted(C.cases()))
def test_configuration_names_every_tensor(name):
    raw = C.cases()[name]
    cfg = registry.from_json(raw).parse(raw)
    w = C.weights(raw)
    assert {k: tuple(v.shape) for k, v in w.items()} == cfg.tensor_shapes()
    check_tensors(cfg, w)
    assert cfg.count_parameters() == sum(v.numel() for v in w.values())
    assert {k: tuple(v.shape) for k, v in random_parameters(cfg).items()} == cfg.tensor_shapes()
    assert [s.weights for s in cfg.layers] == [O.owner(raw, i) for i in range(len(cfg.layers))]


def test_configuration_reads_every_field():
    raw = C.cases()["odd"]
    cfg = LayerListConfig.from_json(json.loads(json.dumps(raw)))
    a, m = cfg.layers[0].mixer, cfg.layers[1].mixer
    assert isinstance(a, AttentionMixer) and (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first) == (6, 2, 24, 40, 37, 3)
    assert a.rot == Rotary(8, 10000.0, False, RotaryScaling(4.0, 1.0, 4.0, 64.0)) and a.sink and a.gate and a.qk_norm
    assert isinstance(m, Mamba2Mixer) and (m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups) == (6, 20, 28, 3, 3, 5)
    assert cfg.layers[3].mlp is None and cfg.layers[0].mlp.ff == 88
    assert (cfg.eps, cfg.logit_softcap, cfg.hidden_size, cfg.vocab_size) == (1e-5, 20.0, 84, 331)
    assert cfg.layers[3].mixer.rot.scaling is None and cfg.layers[3].mixer.keep_first == 0


@pytest.mark.parametrize("change, word", [
    (lambda d: d["layers"][0].update(type="ring"), "unknown layer type"),
    (lambda d: d["layers"][0]["mixer"].update(heads=5), "multiple"),
    (lambda d: d["layers"][0]["mixer"].pop("dim"), "dim"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=26), "exceeds"),
    (lambda d: d["layers"][1]["mixer"].update(norm_groups=7), "norm_groups"),
    (lambda d: d["layers"][1]["mixer"].update(groups=4), "groups"),
    (lambda d: d["layers"][2].update(weights_of=2), "weights_of"),
    (lambda d: d["layers"][2].update(weights_of=0), "other sizes"),
    (lambda d: d["layers"][0]["mlp"].update(kind="sparse"), "kind"),
    (lambda d: d.update(layers=[]), "layers"),
    (lambda d: d.update(vocab=0), "vocab"),
])
def test_configuration_mistakes_are_named(change, word):
    raw = copy.deepcopy(C.cases()["odd"])
    change(raw)
    with pytest.raises(ValueError, match=word):
        LayerListConfig.from_json(raw)


def test_unknown_architecture_is_refused():
    with pytest.raises(ValueError, match="architecture"):
        registry.from_json({"architecture": "nobody"})


def test_engine_class_follows_the_configuration():
    from ghassan_b200.models.config import ModelConfig
    assert registry.engine_class(ModelConfig()).__name__ == "InferenceEngine"
    assert registry.engine_class(LayerListConfig.from_json(C.cases()["odd"])).__name__ == "LayerEngine"


@pytest.mark.parametrize("scaling", [None, C.SCALING, {"factor": 16.0, "low": 2.0, "high": 2.0, "original": 256},
                                     {"factor": 2.5, "low": 0.5, "high": 9.0, "original": 4096}])
def test_rotation_frequencies(scaling):
    rot = {"base": 5e4, "dims": 40, "scaling": scaling}
    got = Rotary.parse(rot).frequencies()
    np.testing.assert_allclose(got, O.rotary_frequencies(rot), rtol=1e-12)
    if scaling:
        plain = O.rotary_frequencies(dict(rot, scaling=None))
        wl = 2 * math.pi / plain
        assert (got[wl < scaling["original"] / scaling["high"]] == plain[wl < scaling["original"] / scaling["high"]]).all()
        assert (got < plain).any()


# ------------------------------------------------------------------------------------------------ files
def test_safetensors_round_trip(tmp_path):
    from ghassan_b200.formats import safetensors as ST
    t = {"a": torch.randn(3, 5).to(torch.bfloat16), "b.c": torch.arange(7, dtype=torch.int32), "e": torch.zeros(0, 4), "s": torch.tensor(2.5)}
    p = str(tmp_path / "m.safetensors")
    ST.save(p, t)
    back = ST.load(p)
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) and back[k].dtype == t[k].dtype for k in t)
    import struct
    head = json.dumps({"__metadata__": {"x": "y"}, "w": {"dtype": "F32", "shape": [2], "data_offsets": [0, 8]}}).encode()
    head += b" " * ((3 - len(head)) % 8)                     # a header that leaves the data unaligned
    (tmp_path / "u.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + struct.pack("<2f", 1.5, -2.0))
    assert ST.load(str(tmp_path / "u.safetensors"))["w"].tolist() == [1.5, -2.0]


@pytest.mark.parametrize("entry", [{"dtype": "F32", "shape": [4], "data_offsets": [0, 8]}, {"dtype": "F32", "shape": [4], "data_offsets": [0, 16]},
                                   {"dtype": "F8", "shape": [8], "data_offsets": [0, 8]}])
def test_safetensors_refuses_what_does_not_fit(tmp_path, entry):
    import struct
    from ghassan_b200.formats import safetensors as ST
    head = json.dumps({"w": entry}).encode()
    (tmp_path / "x.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + b"\0" * 8)
    with pytest.raises(ValueError):
        ST.load(str(tmp_path / "x.safetensors"))


def write_model(folder, name="odd", seed=0):
    from ghassan_b200.formats import safetensors as ST
    raw = C.cases()[name]
    folder.mkdir(exist_ok=True)
    (folder / "config.json").write_text(json.dumps(raw))
    ST.save(str(folder / "model.safetensors"), C.weights(raw, seed))
    return str(folder)


def test_model_folder_loads(tmp_path, capsys):
    from ghassan_b200.cli import infer
    from ghassan_b200.inference import model_io as IO
    path = write_model(tmp_path / "m")
    m = IO.load_model(path)
    assert isinstance(m.cfg, LayerListConfig) and torch.equal(m.named["head"], C.weights(C.cases()["odd"])["head"])
    if not torch.cuda.is_available():
        with pytest.raises(RuntimeError, match="CUDA"):
            IO.build_engine(m)
    assert infer.main(["info", "--model", path]) == 0
    assert "Zikedra" in capsys.readouterr().out


def test_missing_and_misshapen_tensors_are_named():
    cfg = LayerListConfig.from_json(C.cases()["odd"])
    w = C.weights(C.cases()["odd"])
    w.pop("l1.mix.D")
    with pytest.raises(ValueError, match="l1.mix.D"):
        check_tensors(cfg, w)
    w["l1.mix.D"] = torch.zeros(7)
    with pytest.raises(ValueError, match="shape"):
        check_tensors(cfg, w)


# ------------------------------------------------------------------------------------------------ slots
def _slots(name="odd", slots=2, max_len=64, chunk=16):
    from ghassan_b200.inference.layer_cache import SlotManager
    return SlotManager(LayerListConfig.from_json(C.cases()[name]), slots, max_len, chunk, torch.float32, "cpu")


def test_slots_are_given_and_taken_back():
    m = _slots()
    a, b = m.acquire("a"), m.acquire("b")
    assert a != b and m.acquire("a") == a
    with pytest.raises(RuntimeError):
        m.acquire("c")
    m.claim(a, a + 1, 9)
    m.release("a")
    c = m.acquire("c")
    assert c == a and m.length[c] == 0
    with pytest.raises(KeyError):
        m.release("a")


def test_rings_hold_the_window_and_one_portion():
    m = _slots(max_len=4096, chunk=100)
    c = m.layers[0]
    assert c.keep == 3 and c.cap - c.keep >= 37 - 1 + 100 and (c.cap - c.keep) % 128 == 0 and m.limit is None
    short = _slots(max_len=100, chunk=100)
    assert short.limit is not None                        # the ring is shorter than window + portion: length is bounded
    short.claim(0, 1, short.limit)
    with pytest.raises(ValueError, match="exceed"):
        short.claim(0, 1, 1)
    # every position a portion can see has a row of its own
    for p0 in (0, 50, 400, 3000):
        n = 100
        seen = list(range(min(c.keep, p0 + n))) + list(range(max(c.keep, p0 - 37 + 1), p0 + n))
        rows = [p if p < c.keep else c.keep + (p - c.keep) % (c.cap - c.keep) for p in seen]
        assert len(set(rows)) == len(rows)


def test_a_layer_without_a_window_is_bounded_by_max_len():
    raw = copy.deepcopy(C.cases()["odd"])
    for e in (raw["layers"][0], raw["layers"][4]):
        e["mixer"].pop("mask")
    from ghassan_b200.inference.layer_cache import SlotManager
    cfg = LayerListConfig.from_json(raw)
    m = SlotManager(cfg, 1, 200, 16, torch.float32, "cpu")
    assert cfg.layers[0].mixer.window == 0 and m.limit == m.layers[0].cap >= 200


# ------------------------------------------------------------------------------------------------ trace replay
def test_trace_protocol(tmp_path):
    from ghassan_b200.cli import trace

    class Fake:
        def __init__(self):
            self.log = []

        def step(self, key, toks, want):
            self.log.append(("step", key, list(toks)))
            return torch.tensor([[float(toks[w]), 0.5] for w in want]) if want else None

        def check(self, what):
            pass

        def end(self, key):
            self.log.append(("end", key))

    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": [8, 40, 9, 41], "want": [1, 3]}], "end": []}), "",
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": [4], "want": []}], "end": ["a"]})]
    eng, said = Fake(), []
    trace.run(eng, lines, str(tmp_path), said.append)
    assert said == ["done 0", "done 1"] and eng.log == [("step", "a", [8, 40, 9, 41]), ("step", "a", [4]), ("end", "a")]
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [40.0, 0.5, 41.0, 0.5] and not (tmp_path / "1.f32").exists()
    with pytest.raises(SystemExit):
        trace._parser().parse_args(["--model", "m", "--out", "o", "--dtype", "int8"])


# ------------------------------------------------------------------------------------------------ the oracle
def test_oracle_does_not_look_ahead():
    raw = C.cases()["odd"]
    w, ids = C.as_numpy(C.weights(raw, 3)), C.tokens(raw, 50)
    full = O.run(raw, w, ids)
    for n in (1, 7, 38):
        np.testing.assert_allclose(O.run(raw, w, ids[:n]), full[:n], atol=1e-9)


def _mutants():
    def mask(size=0, keep=0):
        def f(raw, w):
            raw["layers"][0]["mixer"]["mask"]["size"] += size
            raw["layers"][0]["mixer"]["mask"]["keep_first"] += keep
        return f

    def sinkless(raw, w):
        w["l0.mix.sink"] = np.full_like(w["l0.mix.sink"], -1e9)

    def ungated(raw, w):
        w["l0.mix.g"] = np.zeros_like(w["l0.mix.g"])

    def unscaled(raw, w):
        raw["layers"][0]["mixer"]["rot"]["scaling"] = None

    def one_tap(raw, w):
        w["l1.mix.conv"] = w["l1.mix.conv"] * np.array([0.0, 1.0])

    def stateless(raw, w):
        w["l1.mix.A_log"] = np.full_like(w["l1.mix.A_log"], 8.0)

    return {"window_in": mask(size=-1), "window_out": mask(size=1), "kept_in": mask(keep=-1), "kept_out": mask(keep=1), "sink": sinkless,
            "gate": ungated, "rotation": unscaled, "convolution": one_tap, "state": stateless}


@pytest.mark.parametrize("kind", sorted(_mutants()))
def test_edge_inputs_show_a_planted_mistake(kind):
    """Each mistake moves the logits at its own places by far more than the GPU tests allow there."""
    raw, w = C.edge_case()
    w = C.as_numpy(w)
    ids, places = C.edge_tokens()
    good = O.run(raw, w, ids)
    raw2, w2 = copy.deepcopy(raw), dict(w)
    _mutants()[kind](raw2, w2)
    d = C.distance(O.run(raw2, w2, ids), good)
    at = places.get(kind, [])
    assert (d[at].min() if at else d.max()) > 0.2, d[at] if at else d.max()


def test_edge_inputs_reach_the_kept_prefix_from_far():
    raw, w = C.edge_case()
    ids, places = C.edge_tokens()
    other = list(ids)
    other[2] = 399
    d = C.distance(O.run(raw, C.as_numpy(w), other), O.run(raw, C.as_numpy(w), ids))
    assert d[places["far"]].min() > 0.2
