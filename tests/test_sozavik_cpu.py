"""Sozavik without a GPU: the configuration read from its own keys and back, the model description (blocks, parts, tensor
names, what the cache manager has to provide), and the plain implementation's mechanisms on cases small enough to check
by hand."""
import json
import math

import pytest
import torch

import plain_sozavik as plain
from tiny_sozavik import SOZAVIKS, make_folder, requests_for

from tiny_llm_infer_b200.config import ConfigError, config_from_dict, describe_model, load_config
from tiny_llm_infer_b200.config.sozavik import SozavikConfig
from tiny_llm_infer_b200.models.model import Model, expected_tensors
from tiny_llm_infer_b200.parts.delta_rule import state_floats
from tiny_llm_infer_b200.parts.position import RotaryHalf, RotaryPairs

F64 = torch.float64


@pytest.mark.parametrize("name", sorted(SOZAVIKS))
def test_config_round_trip(name, tmp_path):
    tiny = SOZAVIKS[name]
    folder = make_folder(tiny, tmp_path)
    raw = json.loads((folder / "config.json").read_text())
    assert raw["architecture"] == "Sozavik"
    cfg = load_config(folder)
    assert isinstance(cfg, SozavikConfig) and cfg == tiny["cfg"]
    assert config_from_dict(cfg.to_dict()).to_dict() == raw


def test_what_may_be_left_out_of_the_configuration():
    raw = SOZAVIKS["Z1"]["cfg"].to_dict()
    m = raw["layers"][3]["mixer"]
    for key in ("softcap", "mask", "v_mix"):
        m[key] = None
    m["rot"]["scaling"] = None
    m["vdim"] = 64                                            # no longer among those that mix
    raw["logit_softcap"] = None
    raw["layers"][3]["mlp"] = None
    got = config_from_dict(raw).layers[3]
    assert got.mixer.softcap is got.mixer.window is got.mixer.rot_scaling is None and got.mixer.v_mix is False
    assert got.mlp is None and config_from_dict(raw).logit_softcap is None
    del m["rot"], m["kv_heads"]
    got = config_from_dict(raw).layers[3].mixer
    assert got.rot_base is None and got.kv_heads == got.heads
    del raw["layers"][1]["mixer"]["vdim"], raw["layers"][4]["mixer"]["v_mix"]
    assert config_from_dict(raw).layers[1].mixer.vdim == 24


def test_description_blocks_and_caches():
    desc = describe_model(SOZAVIKS["Z1"]["cfg"])
    assert [l.block for l in desc.layers] == ["stream_mixer_ffn", "stream_mixer_ffn", "stream_mixer", "stream_mixer_ffn", "stream_mixer"]
    names, _ = expected_tensors(desc)
    assert {"embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.q.norm", "l1.mix.vmix", "l2.mix.norm", "l2.mix.g",
            "l3.mix.q.b", "l3.mix.v.b", "l3.mix.sink", "l3.mix.g", "l3.mix.vmix", "l3.mlp.gate", "l4.mix.k.norm"} <= set(names)
    for absent in ("l0.mix.vmix", "l0.mix.q.b", "l0.mix.sink", "l0.mix.g", "l2.norm2", "l2.mlp.gate", "l3.mix.o.b", "l4.norm2",
                   "lm_head.weight"):
        assert absent not in names, absent
    assert names["l1.mix.q.norm"].shape == (6 * 24,) and names["l1.mix.k.norm"].shape == (2 * 24,)
    assert names["l3.mix.q.norm"].shape == (40,) and names["l3.mix.k.norm"].shape == (40,)
    assert names["l3.mix.g"].shape == (4, 128) and names["l3.mix.vmix"].shape == () and names["l3.mix.v.b"].shape == (80,)
    assert names["l2.mix.q"].shape == (48, 128) and names["l2.mix.v"].shape == names["l2.mix.g"].shape == (72, 128)
    assert names["l2.mix.norm"].shape == (72,) and names["l2.mix.o"].shape == (128, 72)
    model = Model(desc, torch.float32, None)
    needs = model.cache_needs()
    assert sorted(needs) == [0, 1, 2, 3, 4]
    assert needs[0][0].planes == ((4, 32), (4, 16)) and needs[0][0].window == 40 and needs[0][1] is None
    assert needs[1][0].planes == ((2, 24), (2, 40)) and needs[1][0].window == 25
    assert needs[2][0] is None and needs[2][1].shape == (state_floats(3, 3, 16, 24, 1),)
    assert needs[3][0].window == 21 and needs[4][0].window is None
    # the first layer that mixes leaves its values, whichever type it has; the others take them in
    assert [getattr(b.mixers()[0], "value_mix", None) for b in model.blocks] == [None, "first", None, "mix", "mix"]
    other = Model(describe_model(SOZAVIKS["Z2"]["cfg"]), torch.float32, None)
    assert [getattr(b.mixers()[0], "value_mix", None) for b in other.blocks] == [None, "first", "mix", None, "mix"]


def test_config_errors():
    raw = SOZAVIKS["Z1"]["cfg"].to_dict()
    for path, value, text in ((("layers", 0, "type"), "window", "not a mixer"),
                              (("layers", 0, "mixer", "kv_heads"), 3, "multiple of kv_heads"),
                              (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"),
                              (("layers", 0, "mixer", "scale"), None, "scale"),
                              (("layers", 2, "mixer", "decay"), [0.5], "1 numbers for 3 heads"),
                              (("layers", 2, "mixer", "decay"), 0.5, "one number per head"),
                              (("layers", 2, "mixer", "dim"), 0, "dim"),
                              (("layers", 3, "mixer", "softcap"), -1.0, "softcap"),
                              (("layers", 3, "mixer", "rot", "dims"), 42, "rot.dims"),
                              (("layers", 3, "mixer", "rot", "dims"), 7, "rot.dims"),
                              (("layers", 3, "mixer", "rot", "base"), None, "base"),
                              (("layers", 3, "mixer", "rot", "scaling", "factor"), 0.0, "factor"),
                              (("layers", 3, "mixer", "rot", "scaling", "high"), 0.5, "below low"),
                              (("layers", 3, "mixer", "vdim"), 32, "mixes values"),
                              (("layers", 0, "mlp", "kind"), "moe", "not 'dense'"),
                              (("layers", 0, "mlp", "ff"), 0, "ff"),
                              (("logit_softcap",), -2.0, "logit_softcap"),
                              (("norm", "eps"), 0.0, "norm.eps")):
        bad = json.loads(json.dumps(raw))
        at = bad
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(ConfigError, match=text):
            config_from_dict(bad)


def test_parts_refuse_what_they_cannot_do():
    from tiny_llm_infer_b200.parts.registry import lookup
    from tiny_llm_infer_b200.parts.spec import PartSpec
    common = dict(hidden_size=16, q_heads=2, kv_heads=1, key_dim=8, value_dim=8, scale=1.0, dtype=torch.float32, device=None)
    attention = lookup("mixer", "biased_attention")
    with pytest.raises(ValueError, match="is a norm"):
        attention(**common, norm_whole=True)
    with pytest.raises(ValueError, match="value_mix"):
        attention(**common, value_mix="second")
    with pytest.raises(ValueError, match="values that are keys"):
        attention(**common, values_are_keys=True, value_mix="mix")
    part = attention(**common, value_mix="mix")

    class Ctx:
        memo = {}
    with pytest.raises(ValueError, match="has left its values"):
        part._value_mix(torch.zeros(1, 32), Ctx)
    with pytest.raises(ValueError, match="decays"):
        lookup("mixer", "fixed_decay")(hidden_size=16, heads=2, key_dim=8, value_dim=8, decays=(0.5,), norm_eps=1e-5,
                                       dtype=torch.float32, device=None)
    with pytest.raises(ValueError, match="neighbouring"):
        lookup("mixer", "gq_attention")(hidden_size=16, q_heads=2, kv_heads=1, head_dim=8, dtype=torch.float32, device=None,
                                        position=PartSpec("rotary_pairs", dict(head_dim=8, theta=100.0)))
    with pytest.raises(ValueError, match="factor"):
        RotaryPairs(8, 100.0, torch.float32, None, scaling=dict(factor=0.0, low=1.0, high=2.0, original=10.0))


@pytest.mark.parametrize("dims,base,scaling", [(16, 500.0, (4.0, 1.0, 4.0, 64.0)), (6, 77.0, (8.0, 1.5, 3.0, 40.0)),
                                               (128, 1e6, (16.0, 2.0, 2.0, 4096.0)), (32, 1e4, None)])
def test_scaled_frequencies(dims, base, scaling):
    s = None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))
    for cls in (RotaryHalf, RotaryPairs):
        part = cls(dims, base, torch.float32, None, scaling=s)
        freq, width = part.fused_rotary()
        want = plain.frequencies(dims, base, s)
        assert width == dims and torch.allclose(freq.double(), torch.tensor(want, dtype=F64), rtol=2e-7)
    if s is not None:
        raw = plain.frequencies(dims, base, None)
        ratio = [a / b for a, b in zip(want, raw)]
        assert ratio[0] == 1.0 and abs(ratio[-1] - 1.0 / s["factor"]) < 1e-12     # fast ones stay, slow ones are divided
        assert all(a >= b - 1e-12 for a, b in zip(ratio, ratio[1:]))


def test_rotation_and_scaling_by_hand():
    f = plain.frequencies(4, 100.0, None)
    assert f == [1.0, 0.1]
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]] * 3, dtype=F64)
    got = plain.rotate_pairs(x, f)
    c, s, c1, s1 = math.cos(2), math.sin(2), math.cos(0.2), math.sin(0.2)
    assert torch.allclose(got[2, 0], torch.tensor([c - 2 * s, 2 * c + s, 3 * c1 - 4 * s1, 4 * c1 + 3 * s1, 5.0], dtype=F64))
    assert torch.equal(got[0], x[0])
    # wavelengths 2 pi (turns 10 / 2 pi = 1.59 within ten tokens) and 20 pi (0.159): kept, divided, blended
    sc = lambda low, high: dict(factor=4.0, low=low, high=high, original=10.0)
    assert plain.frequencies(4, 100.0, sc(0.5, 1.0)) == [1.0, 0.025]
    blend = (10.0 / (2 * math.pi) - 1.0) / 2.0
    assert math.isclose(plain.frequencies(4, 100.0, sc(1.0, 3.0))[0], (1 - blend) / 4 + blend)


def test_attention_by_hand():
    # two tokens, one head, keys of one element; the window, the cap and the sink one by one
    q = torch.tensor([[[1.0]], [[2.0]], [[1.0]]], dtype=F64)
    k = torch.tensor([[[1.0]], [[0.5]], [[-1.0]]], dtype=F64)
    v = torch.eye(3, dtype=F64).view(3, 1, 3)
    e = math.exp
    got = plain.softmax_attention(q, k, v, 1.0, None, None, None)
    assert torch.allclose(got[1, 0], torch.tensor([e(2) / (e(2) + e(1)), e(1) / (e(2) + e(1)), 0.0], dtype=F64))
    got = plain.softmax_attention(q, k, v, 1.0, None, 2, None)              # the third token sees itself and the one before
    assert torch.allclose(got[2, 0], torch.tensor([0.0, e(0.5) / (e(0.5) + e(-1)), e(-1) / (e(0.5) + e(-1))], dtype=F64))
    got = plain.softmax_attention(q, k, v, 3.0, 2.0, 1, torch.tensor([0.7], dtype=F64))
    s = 2.0 * math.tanh(3.0 / 2.0)
    assert torch.allclose(got[0, 0], torch.tensor([e(s) / (e(s) + e(0.7)), 0.0, 0.0], dtype=F64))
    assert torch.equal(plain.mixed_values(v, None, torch.tensor(0.25, dtype=F64)), v)
    assert torch.allclose(plain.mixed_values(v, 2 * v, torch.tensor(0.25, dtype=F64)), 1.25 * v)


def test_norms_gate_and_biases_by_hand():
    m = dict(heads=2, kv_heads=1, dim=1, vdim=1, scale=1.0)
    eye, x = torch.eye(2, dtype=F64), torch.tensor([[3.0, 4.0]], dtype=F64)
    w = {"q": eye, "k": eye[:1], "v": eye[1:], "o": eye, "q.norm": torch.ones(2, dtype=F64), "k.norm": torch.ones(1, dtype=F64)}
    # one token: the softmax gives its own value to both heads
    out, v = plain.whole_normed_attention(x, w, "", m, 1e-9)
    assert torch.allclose(out, torch.tensor([[4.0, 4.0]], dtype=F64)) and torch.equal(v, torch.tensor([[[4.0]]], dtype=F64))
    # the two queries are normed together, so their lengths keep their ratio; the keys, one head alone, come out as +-1
    two = torch.cat([torch.tensor([[-3.0, 4.0]], dtype=F64), torch.tensor([[4.0, 3.0]], dtype=F64)])
    out, _ = plain.whole_normed_attention(two, w, "", m, 1e-12)
    q = [4.0 / math.sqrt(12.5), 3.0 / math.sqrt(12.5)]
    want = [(4.0 * math.exp(-s) + 3.0 * math.exp(s)) / (math.exp(s) + math.exp(-s)) for s in q]
    assert torch.allclose(out[1], torch.tensor(want, dtype=F64))
    w.update({"q.b": torch.zeros(2, dtype=F64), "k.b": torch.zeros(1, dtype=F64), "v.b": torch.tensor([1.0], dtype=F64),
              "q.norm": torch.ones(1, dtype=F64), "sink": torch.tensor([-1e9, 1.0], dtype=F64), "g": torch.zeros(2, 2, dtype=F64)})
    w["g"][1] = torch.tensor([1.0, 0.0], dtype=F64)
    out, v = plain.rotated_attention(x, w, "", m, 1e-9)
    second = math.exp(1.0) / (math.exp(1.0) + math.exp(1.0))                # score one beside a sink of one
    want = torch.tensor([[5.0 * 0.5, 5.0 * second / (1 + math.exp(-3.0))]], dtype=F64)
    assert torch.allclose(out, want) and torch.equal(v, torch.tensor([[[5.0]]], dtype=F64))


def test_recurrence_and_feed_forward_by_hand():
    q = torch.tensor([[[1.0, 0.0]], [[1.0, 2.0]]], dtype=F64)
    k = torch.tensor([[[2.0, 1.0]], [[0.0, 3.0]]], dtype=F64)
    v = torch.tensor([[[5.0]], [[7.0]]], dtype=F64)
    got = plain.fixed_decay_recurrence(q, k, v, [0.5])
    assert torch.equal(got.flatten(), torch.tensor([10.0, 0.5 * 5.0 * (2.0 + 2.0) + 7.0 * 6.0], dtype=F64))
    eye = torch.eye(2, dtype=F64)
    w = {n: eye for n in "qkvgo"}
    w["norm"] = torch.tensor([2.0, 3.0], dtype=F64)
    x = torch.tensor([[1.0, -2.0]], dtype=F64)
    sig = lambda z: 1 / (1 + math.exp(-z))
    a, b = sig(1.0), -2.0 * sig(-2.0)                                       # two heads of one channel: o = silu(x)^3
    o = torch.tensor([a ** 3, b ** 3], dtype=F64)
    want = o / torch.sqrt((o * o).mean()) * w["norm"] * torch.tensor([sig(1.0), sig(-2.0)], dtype=F64)
    assert torch.allclose(plain.lightning(x, w, "", dict(heads=2, dim=1, vdim=1, decay=[0.1, 0.2]), 1e-15)[0], want)
    w = {"gate": eye, "up": torch.tensor([[0.0, 1.0], [1.0, 0.0]], dtype=F64), "down": eye}
    assert torch.equal(plain.relu_unit(x, w, "")[0], torch.tensor([-2.0, 0.0], dtype=F64))


@pytest.mark.parametrize("name", sorted(SOZAVIKS))
def test_a_missing_mechanism_would_show(name, tmp_path):
    """The weights of the tiny models make every mechanism matter: the plain implementation with another constant,
    without a bias, a gate, a sink or the mixing, with a window one token off or without the first tokens moves the
    logits far beyond the tolerances of the comparisons with the engine."""
    import numpy as np
    from tiny_llm_infer_b200.weights.safetensors_io import SafetensorsFile
    tiny = SOZAVIKS[name]
    folder = make_folder(tiny, tmp_path)
    cfg = json.loads((folder / "config.json").read_text())
    f = SafetensorsFile(folder / "model.safetensors")
    w = {n: f.read(n).clone() for n in f.tensors}
    f.close()
    toks = max(requests_for(tiny).values(), key=len)[-120:]
    ref = plain.forward(cfg, w, toks).numpy()

    def moved(changed_cfg=None, changed_w=None, tokens=None):
        got = plain.forward(changed_cfg or cfg, changed_w or w, tokens or toks).numpy()
        d = got[-40:] - ref[-40:]
        return float((np.sqrt(((d - d.mean(1, keepdims=True)) ** 2).mean(1)) / ref[-40:].std(1)).max())

    def with_weights(fn):
        return {k: fn(k, v) for k, v in w.items()}

    floor = 2e-3
    for suffix in (".q.b", ".k.b", ".v.b", ".mix.g", ".vmix"):
        if any(k.endswith(suffix) for k in w):
            assert moved(changed_w=with_weights(lambda k, v: torch.zeros_like(v) if k.endswith(suffix) else v)) > floor, suffix
    if any(k.endswith(".sink") for k in w):
        assert moved(changed_w=with_weights(lambda k, v: v - 30.0 if k.endswith(".sink") else v)) > floor
    if any(k.endswith(".q.norm") for k in w):
        assert moved(changed_w=with_weights(lambda k, v: v.flip(0) if k.endswith(".q.norm") else v)) > floor
    for path, change in ((("mixer", "scale"), lambda v: v * 1.5), (("mixer", "softcap"), lambda v: v * 0.3),
                         (("mixer", "mask", "size"), lambda v: v + 1), (("mixer", "mask", "size"), lambda v: v - 1),
                         (("mixer", "rot", "base"), lambda v: v * 3.0), (("mixer", "rot", "dims"), lambda v: v - 2),
                         (("mixer", "rot", "scaling"), lambda v: None), (("mixer", "rot", "scaling", "original"), lambda v: v * 3),
                         (("mixer", "v_mix"), lambda v: False), (("mixer", "decay"), lambda v: [a * 0.9 for a in v])):
        changed = json.loads(json.dumps(cfg))
        for layer in changed["layers"]:
            d = layer
            for key in path[:-1]:
                d = d.get(key) or {}
            if d.get(path[-1]) is not None:
                d[path[-1]] = change(d[path[-1]])
        if changed != cfg:
            assert moved(changed_cfg=changed) > floor, path
    if cfg.get("logit_softcap"):
        assert moved(changed_cfg=dict(cfg, logit_softcap=cfg["logit_softcap"] * 2)) > floor
    assert moved(tokens=toks[40:]) > floor                       # the first forty tokens forgotten
