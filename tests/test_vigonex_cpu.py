"""Vigonex without a GPU: the configuration read from its own keys and back, the model description (blocks, parts, tensor
names, what the cache manager has to provide), and the plain implementation's mechanisms on cases small enough to check
by hand."""
import json
import math

import pytest
import torch

import plain_vigonex as plain
from tiny_vigonex import VIGONEXES, as_read, make_folder, requests_for

from tiny_llm_infer_b200.config import ConfigError, config_from_dict, describe_model, load_config
from tiny_llm_infer_b200.config.vigonex import VigonexConfig
from tiny_llm_infer_b200.models.model import Model, expected_tensors
from tiny_llm_infer_b200.parts.delta_rule import state_floats

F64 = torch.float64


@pytest.mark.parametrize("name", sorted(VIGONEXES))
def test_config_round_trip(name, tmp_path):
    tiny = VIGONEXES[name]
    folder = make_folder(tiny, tmp_path)
    raw = json.loads((folder / "config.json").read_text())
    assert raw["architecture"] == "Vigonex"
    assert config_from_dict(raw) == as_read(tiny["cfg"])
    cfg = load_config(folder)                                # the ranks come from the tensors' shapes
    assert isinstance(cfg, VigonexConfig) and cfg == tiny["cfg"]
    assert config_from_dict(cfg.to_dict()).to_dict() == raw


def test_description_blocks_and_caches():
    tiny = VIGONEXES["G1"]
    desc = describe_model(tiny["cfg"])
    assert [l.block for l in desc.layers] == ["hyper_mixer_ffn_gated_shifted", "hyper_mixer_ffn_gated_shifted",
                                              "hyper_mixer_gated_shifted", "hyper_mixer_ffn_gated_shifted"]
    names, _ = expected_tensors(desc)
    assert {"embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.shift", "l0.rg1", "l0.rg1.b", "l0.rg2.b", "l0.hc1.in",
            "l0.hc1.out", "l0.hc2.mix", "l0.mix.q.b", "l0.mix.o.b", "l0.mix.lq1", "l0.mix.lk2", "l0.mlp.router",
            "l0.mlp.e5.gate", "l0.mlp.shared.sg", "l1.mix.r", "l1.mix.a.b", "l1.mix.w0", "l1.mix.norm", "l1.mlp.gate",
            "l3.mlp.e4.down"} <= set(names)
    for absent in ("l2.norm2", "l2.hc2.in", "l2.rg2", "l3.mlp.shared.sg", "l3.mlp.shared.gate", "l0.mix.g", "l1.mix.q",
                   "lm_head.weight", "l0.mlp.e6.up"):
        assert absent not in names, absent
    assert names["l0.mix.q"].shape == (6 * 2 * 24, 128) and names["l0.mix.k"].shape == (2 * 2 * 24, 128)
    assert names["l0.mix.v"].shape == (2 * 40, 128) and names["l0.mix.o"].shape == (128, 6 * 40)
    assert names["l0.hc1.mix"].shape == (3, 3) and names["l0.mix.lq1"].shape == (24,)
    assert names["l1.mix.w1"].shape == (8, 128) and names["l1.mix.w2"].shape == (64, 8) and names["l1.mix.norm"].shape == (64,)
    model = Model(desc, torch.float32, None)
    needs = model.cache_needs()
    assert sorted(needs) == list(range(8))                   # per layer the shift's state, then the mixer's cache or state
    for shift in (0, 2, 4, 6):
        assert needs[shift][0] is None and needs[shift][1].shape == (128,)
    assert needs[1][0].planes == ((2, 48), (2, 40)) and needs[1][1] is None
    assert needs[3][0] is None and needs[3][1].shape == (state_floats(4, 4, 16, 16, 1),)
    assert needs[5][0].planes == ((3, 32), (3, 16)) and needs[7][1].shape == (state_floats(2, 2, 40, 40, 1),)
    # two tensors of streams, before and after an update, are counted beside the widest part
    assert model.workspace_floats(10, 1) > 10 * 2 * 3 * 128


def test_config_errors():
    raw = VIGONEXES["G1"]["cfg"].to_dict()
    for path, value, text in ((("layers", 0, "type"), "window", "not a mixer"),
                              (("layers", 0, "mixer", "kv_heads"), 4, "multiple of kv_heads"),
                              (("layers", 0, "mixer", "softcap"), -1.0, "softcap"),
                              (("layers", 0, "mixer", "q_temp", "every"), 0, "q_temp.every"),
                              (("layers", 0, "mixer", "diff"), None, "diff"),
                              (("layers", 1, "mixer", "dim"), 0, "dim"),
                              (("layers", 0, "mlp", "kind"), "sparse", "neither"),
                              (("layers", 0, "mlp", "router", "top"), 7, "router.top"),
                              (("layers", 0, "mlp", "expert", "limit"), 0.0, "expert_limit"),
                              (("layers", 0, "mlp", "shared", "limit"), -2.0, "shared_limit"),
                              (("streams",), 0, "streams"),
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
    common = dict(hidden_size=16, q_heads=2, kv_heads=1, key_dim=8, value_dim=8, scale=1.0, dtype=torch.float32, device=None,
                  differential=(0.5, 1e-6))
    attention = lookup("mixer", "biased_attention")
    attention(**common)
    with pytest.raises(ValueError, match="two maps"):
        attention(**common, unit_norm_eps=1e-5)
    with pytest.raises(ValueError, match="eps"):
        attention(**dict(common, differential=(0.5, 0.0)))
    moe = lookup("feed_forward", "moe")
    with pytest.raises(ValueError, match="shared unit"):
        moe(hidden_size=16, experts=4, top=1, expert_size=8, dtype=torch.float32, device=None, weight_on="output",
            router_scores="softmax_all", shared_gate="sg")
    with pytest.raises(ValueError, match="softmax over the chosen"):
        moe(hidden_size=16, experts=4, top=1, expert_size=8, dtype=torch.float32, device=None, weight_on="output",
            router_scores="softmax", router_scale=2.0)
    with pytest.raises(ValueError, match="wider"):
        lookup("mixer", "erase_delta")(hidden_size=16, heads=1, key_dim=600, value_dim=8, decay_rank=4, norm_eps=1e-5,
                                       dtype=torch.float32, device=None)
    block = lookup("block", "hyper_mixer")
    parts = {r: lookup("norm", "stream_mix")(streams=2, dtype=torch.float32, device=None) for r in block.roles}
    with pytest.raises(TypeError, match="several streams"):
        block(parts).forward(torch.zeros(1, 4), torch.zeros(1, 4), None, None)
    assert PartSpec("stream_norm").kind == "stream_norm"


def test_streams_shift_and_sinusoids_by_hand():
    xs = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=F64)                         # two streams, one token
    assert torch.equal(plain.read_streams(xs, torch.tensor([3.0, -1.0], dtype=F64)), torch.tensor([[-7.0, -14.0]], dtype=F64))
    # mix is [from, to]: stream 0 goes to stream 1 only, stream 1 to both
    mix = torch.tensor([[0.0, 1.0], [0.5, 2.0]], dtype=F64)
    got = plain.write_streams(xs, mix, torch.tensor([1.0, -2.0], dtype=F64), torch.tensor([[100.0, 0.0]], dtype=F64))
    assert torch.equal(got, torch.tensor([[[5.0 + 100.0, 10.0]], [[1.0 + 20.0 - 200.0, 2.0 + 40.0]]], dtype=F64))
    h = torch.tensor([[1.0, 1.0], [3.0, 5.0], [0.0, 2.0]], dtype=F64)
    got = plain.token_shift(h, torch.tensor([0.5, 1.0], dtype=F64))
    assert torch.equal(got, torch.tensor([[0.5, 0.0], [2.0, 1.0], [1.5, 5.0]], dtype=F64))
    pos = plain.sinusoids(4, 5, F64)
    f1 = 10000.0 ** (-2.0 / 5)
    f2 = 10000.0 ** (-4.0 / 5)
    assert torch.allclose(pos[3], torch.tensor([math.sin(3), math.cos(3), math.sin(3 * f1), math.cos(3 * f1), math.sin(3 * f2)], dtype=F64))
    assert torch.equal(pos[0], torch.tensor([0.0, 1.0, 0.0, 1.0, 0.0], dtype=F64))


def test_temperature_experts_and_router_by_hand():
    t = plain.query_temperature(8, 0.5, 3, F64)
    want = [1.0, 1.0] + [1 + 0.5 * math.log(2.0)] * 3 + [1 + 0.5 * math.log(3.0)] * 3
    assert torch.allclose(t, torch.tensor(want, dtype=F64))
    eye = torch.eye(2, dtype=F64)
    # gate 3 is held at 1.5, up -4 at -1.5; gate -4 is not held (only from above), up 1 not either
    got = plain.clamped_expert(torch.tensor([[1.0, 0.0]], dtype=F64), torch.tensor([[3.0, 0.0], [-4.0, 0.0]], dtype=F64),
                               torch.tensor([[-4.0, 0.0], [1.0, 0.0]], dtype=F64), eye, 1.5)
    sig = lambda v: 1 / (1 + math.exp(-v))
    assert torch.allclose(got, torch.tensor([[1.5 * sig(1.702 * 1.5) * -0.5, -4.0 * sig(1.702 * -4.0) * 2.0]], dtype=F64))
    z = torch.tensor([[0.3, 2.0, -1.0, 1.0]], dtype=F64)
    chosen, weights = plain.route(torch.eye(4, dtype=F64)[:1], z.T @ torch.eye(4, dtype=F64)[:1], 2, 2.5)
    s = torch.softmax(z[0], 0)
    assert chosen[0].tolist() == [1, 3] and torch.allclose(weights[0], 2.5 * s[[1, 3]])
    assert torch.allclose(plain.router_margin(torch.eye(4, dtype=F64)[:1], z.T @ torch.eye(4, dtype=F64)[:1], 2), torch.tensor([0.7], dtype=F64))


def test_difference_of_maps_and_delta_rule_by_hand():
    # one head, maps of one element, values of one element: the second token weighs two values per map
    m = dict(heads=1, kv_heads=1, dim=1, vdim=2, scale=1.0, diff=0.25)
    w = {k: torch.zeros(s, dtype=F64) for k, s in (("q", (2, 2)), ("q.b", (2,)), ("k", (2, 2)), ("k.b", (2,)), ("v", (2, 2)),
                                                   ("v.b", (2,)), ("o", (2, 2)), ("o.b", (2,)))}
    w["q.b"] = torch.tensor([1.0, 2.0], dtype=F64)
    w["k"] = torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=F64)                            # map 1 sees x_0, map 2 x_1
    w["v"], w["o"], w["o.b"] = torch.eye(2, dtype=F64), torch.eye(2, dtype=F64), torch.tensor([0.5, 0.0], dtype=F64)
    for n, v in (("lq1", 0.5), ("lk1", 0.6), ("lq2", 0.2), ("lk2", -1.0)):
        w[n] = torch.tensor([v], dtype=F64)
    x = torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=F64)
    got = plain.differential_attention(x, w, "", m, 1e-12)
    lam = math.exp(0.3) - math.exp(-0.2) + 0.25
    a1 = math.exp(1.0) / (math.exp(1.0) + 1.0)                                            # map 1: scores 1, 0
    a2 = 1.0 / (1.0 + math.exp(2.0))                                                      # map 2: scores 0, 2
    o = torch.tensor([a1 - lam * a2, (1 - a1) - lam * (1 - a2)], dtype=F64)
    want = o / torch.sqrt((o * o).mean()) * 0.75 + torch.tensor([0.5, 0.0], dtype=F64)
    assert torch.allclose(got[1], want, atol=1e-9)
    # the delta rule, one head of two channels: the second token removes along its unit key from the state before the decay
    m = dict(heads=1, dim=2)
    eye = torch.eye(2, dtype=F64)
    w = dict(r=eye, k=eye, v=2.0 * eye, w1=torch.zeros(1, 2, dtype=F64), w2=torch.zeros(2, 1, dtype=F64),
             w0=torch.tensor([0.0, 1.0], dtype=F64), a=torch.zeros(2, 2, dtype=F64), g=torch.zeros(2, 2, dtype=F64),
             norm=torch.tensor([1.0, 3.0], dtype=F64), o=eye)
    w["a.b"] = torch.tensor([0.0, 2.0], dtype=F64)
    x = torch.tensor([[3.0, 4.0], [1.0, 0.0]], dtype=F64)
    got = plain.general_delta(x, w, "", m, 1e-12)
    sig = lambda v: 1 / (1 + math.exp(-v))
    S = torch.outer(x[0], 2.0 * x[0])
    d = torch.tensor([math.exp(-math.exp(-0.5) * sig(0.0)), math.exp(-math.exp(-0.5) * sig(1.0))], dtype=F64)
    a = torch.tensor([sig(0.0), sig(2.0)], dtype=F64)
    u = x[1] / math.sqrt(1 + 1e-6)
    S = d.unsqueeze(1) * S - torch.outer(a * u, u @ S) + torch.outer(x[1], 2.0 * x[1])
    o = S.T @ x[1]
    want = o / torch.sqrt((o * o).mean()) * w["norm"] * 0.5
    assert torch.allclose(got[1], want, atol=1e-9)


@pytest.mark.parametrize("name", sorted(VIGONEXES))
def test_a_missing_mechanism_would_show(name, tmp_path):
    """The weights of the tiny models make every mechanism matter: the plain implementation with another constant,
    without a bias, a gate, the shift, the mix or the difference, or without the first tokens moves the logits far
    beyond the tolerances of the comparisons with the engine."""
    import numpy as np
    from tiny_llm_infer_b200.weights.safetensors_io import SafetensorsFile
    tiny = VIGONEXES[name]
    folder = make_folder(tiny, tmp_path)
    cfg = json.loads((folder / "config.json").read_text())
    f = SafetensorsFile(folder / "model.safetensors")
    w = {n: f.read(n).clone() for n in f.tensors}
    f.close()
    toks = max(requests_for(tiny).values(), key=len)[:120]
    ref = plain.forward(cfg, w, toks).numpy()

    def moved(changed_cfg=None, changed_w=None, tokens=None):
        got = plain.forward(changed_cfg or cfg, changed_w or w, tokens or toks).numpy()
        d = got[-40:] - ref[-40:]
        return float((np.sqrt(((d - d.mean(1, keepdims=True)) ** 2).mean(1)) / ref[-40:].std(1)).max())

    def with_weights(fn):
        return {k: fn(k, v) for k, v in w.items()}

    floor = 2e-3
    for suffix in (".q.b", ".v.b", ".o.b", "mix.a.b", ".w0", ".w2", ".shift", "rg1.b", "rg2.b", "lq1", "lk2", ".sg", ".rg1", ".rg2"):
        if any(k.endswith(suffix) for k in w):
            assert moved(changed_w=with_weights(lambda k, v: torch.zeros_like(v) if k.endswith(suffix) else v)) > floor, suffix
    if cfg["streams"] > 1:
        assert moved(changed_w=with_weights(lambda k, v: v.T.contiguous() if k.endswith(".mix") else v)) > floor
        assert moved(changed_w=with_weights(lambda k, v: v.flip(0) if k.endswith("hc1.in") else v)) > floor
    # a mean bias on the keys of a map changes nothing a softmax sees unless the temperature or the cap tells apart
    for path, f_ in ((("mixer", "scale"), lambda v: v * 1.5), (("mixer", "softcap"), lambda v: v * 0.3),
                     (("mixer", "diff"), lambda v: v + 0.1), (("mixer", "q_temp", "coef"), lambda v: v * 2),
                     (("mixer", "q_temp", "every"), lambda v: v + 1), (("mlp", "expert", "limit"), lambda v: v * 0.7),
                     (("mlp", "router", "scale"), lambda v: v * 1.2), (("mlp", "shared", "limit"), lambda v: v * 0.7),
                     (("mlp", "router", "top"), lambda v: v - 1 if v > 1 else v)):
        changed = json.loads(json.dumps(cfg))
        for layer in changed["layers"]:
            d = layer
            for key in path[:-1]:
                d = d.get(key) or {}
            if d.get(path[-1]) is not None:
                d[path[-1]] = f_(d[path[-1]])
        if changed != cfg:
            assert moved(changed_cfg=changed) > floor, path
    for key, value in (("embedding", {"scale": cfg["embedding"]["scale"] * 1.3}), ("logit_scale", cfg["logit_scale"] * 1.1)):
        assert moved(changed_cfg=dict(cfg, **{key: value})) > floor, key
    assert moved(tokens=toks[40:]) > floor                       # the first forty tokens forgotten
