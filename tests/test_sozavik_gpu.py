"""Sozavik on the GPU against the plain implementation (``plain_sozavik.py``).

Each mechanism alone, as the registered part or kernel with sizes of its own: both attentions over scrambled pages that
hold other requests' leftovers, with inputs shaped so that single keys at the window's edge (the last one inside and the
first one outside), at page borders and next to the query stand out, with and without another layer's values mixed in;
long requests whose keys are dealt to several blocks; the recurrence with constant decays, whole, in portions down to one
token, side by side and in slots that are used again, with heads slow enough that the first tokens still show at the end;
ReLU units on every product kernel.  Then whole models through ``bin/trace_run`` in every way of cutting, the first tokens
one by one, long decoding, and greedy generation through the engine's entry point under budgets and starved pools.

Tolerances, as a row's root-mean-square difference (its mean taken off) over the row's own spread: float32 2e-5
against the plain implementation and between the ways of cutting; bfloat16 about three times what a B200 shows per
configuration."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import plain_sozavik as plain
import replay
from test_tetodra_gpu import (Bench, build_part, make_ctx, read_model, recurrence_run, relative_rows, run_tool, turn,
                              whole_then_portions)
from tiny_sozavik import SOZAVIKS, make_folder, prompt, requests_for

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda:0"
F64 = torch.float64


# ----------------------------------------------------------------------------- the two attentions as parts
def edge_inputs(lengths, hidden, window, page, seed):
    """Random rows in which chosen queries are the turned row (``turn``) of one key: by turns the last key inside their
    window, the first one outside it, the keys on both sides of a page's border inside it, the first token, and the key
    next to the query.  With keys projected like the first query head of their group after the same turn, that one score
    stands out among all others."""
    g = torch.Generator().manual_seed(seed)
    R = turn(hidden)
    xs = []
    for L in lengths:
        x = torch.randn(L, hidden, generator=g)
        queries, i, k = set(), 3, 0
        while i < L:
            w = window or i + 1
            border = i // page * page
            j = [i - w + 1, i - w, border, i - 1, border - 1, 0, 1][k % 7]
            if 0 <= j < i and j not in queries:
                x[i] = R @ x[j]
                queries.add(i)
            k += 1
            i += 2 + k % 3 % 2
        xs.append(x)
    return xs


def tie(H, G, dk, hidden):
    R = turn(hidden)

    def change(w):
        for kv in range(G):
            first = kv * (H // G)
            w["k"][kv * dk:(kv + 1) * dk] = w["q"][first * dk:(first + 1) * dk] @ R
    return change


class WithOtherValues:
    """A part that mixes, behind a stand-in for the layer that leaves its values: a product with a matrix of its own in
    a tensor of wider rows."""

    def __init__(self, part, matrix, bias, extra):
        self.part, self.matrix, self.bias, self.extra = part, matrix, bias, extra

    def cache_spec(self):
        return self.part.cache_spec()

    def state_spec(self):
        return self.part.state_spec()

    def forward(self, x, ctx, cache):
        values = x.to(torch.float32) @ self.matrix.to(torch.float32).T
        rows = torch.full((x.shape[0], values.shape[1] + self.extra), 7.0, dtype=x.dtype, device=x.device)
        rows[:, self.extra // 2:self.extra // 2 + values.shape[1]] = values.to(x.dtype)
        ctx.memo[self.part.FIRST_VALUES] = (rows[:, self.extra // 2:self.extra // 2 + values.shape[1]], self.bias)
        return self.part.forward(x, ctx, cache)


def other_values(part, rows, hidden, dtype, biased, extra, seed):
    g = torch.Generator().manual_seed(seed)
    matrix = (torch.randn(rows, hidden, generator=g) * 0.3).to(dtype)
    bias = torch.randn(rows, generator=g) if biased else None
    wrapped = WithOtherValues(part, matrix.to(DEV), None if bias is None else bias.to(DEV), extra)

    def first(x):
        v = (x.double() @ matrix.double().T).to(dtype).double()
        return v if bias is None else v + bias.double()
    return wrapped, first


def check_edges(fn, window, x, want):
    """The rows' answers hang on the window: one token more or less and some answer moves a lot."""
    if window is not None and window > 1 and x.shape[0] > window + 8:
        for other in (window + 1, window - 1):
            assert (fn(x, other) - want).abs().max() > 0.05 * want.abs().max(), other


ROTATED_CASES = [dict(H=6, G=3, dk=40, dv=24, scale=0.25, cap=9.0, window=37, rot=(500.0, 16), page=16, mix="vec"),
                 dict(H=3, G=1, dk=10, dv=6, scale=0.9, cap=5.0, window=5, rot=(77.0, 4), page=8, mix="odd"),
                 dict(H=4, G=2, dk=128, dv=128, scale=0.09, cap=None, window=100, rot=(1e5, 20), page=32, mix=None),
                 dict(H=5, G=5, dk=12, dv=20, scale=0.5, cap=20.0, window=None, rot=(1e4, 12), page=16, mix="plain"),
                 dict(H=8, G=2, dk=80, dv=176, scale=0.12, cap=30.0, window=64, rot=(1e6, 8), page=16, mix="vec"),
                 dict(H=16, G=1, dk=64, dv=48, scale=0.2, cap=15.0, window=17, rot=(300.0, 2), page=16, mix="vec"),
                 dict(H=1, G=1, dk=24, dv=40, scale=0.4, cap=None, window=1, rot=None, page=16, mix="plain"),
                 dict(H=4, G=4, dk=160, dv=32, scale=0.1, cap=12.0, window=33, rot=(1e4, 36), page=16, mix=None)]


@pytest.mark.parametrize("case", ROTATED_CASES, ids=lambda c: f"h{c['H']}g{c['G']}k{c['dk']}v{c['dv']}w{c['window']}")
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_rotated_attention(case, dtype):
    """Biases, a norm per head, turning pairs with scaled frequencies, cap, window, learned sink, a gate per head, mixing."""
    from tiny_llm_infer_b200.engine.runner import strict_float32
    from tiny_llm_infer_b200.parts.spec import PartSpec
    strict_float32()
    H, G, dk, dv, hidden, mix = case["H"], case["G"], case["dk"], case["dv"], 104, case["mix"]
    scaling = dict(factor=4.0, low=1.0, high=5.0, original=48.0)
    params = dict(hidden_size=hidden, q_heads=H, kv_heads=G, key_dim=dk, value_dim=dv, scale=case["scale"], unit_norm_eps=2e-6,
                  qk_gains=True, softcap=case["cap"], window=case["window"], biases=True, output_bias=False, sink=True,
                  learned_sink=True, output_gate=True, gate_per_head=True, value_mix=None if mix is None else "mix")
    if case["rot"]:
        params["position"] = PartSpec("rotary_pairs", dict(head_dim=dk, theta=case["rot"][0], rotary_dim=case["rot"][1],
                                                           scaling=scaling))

    def change(w):
        tie(H, G, dk, hidden)(w)
        for n in ("q.b", "k.b"):
            w[n] *= 0.6
        for n in ("q.norm", "k.norm"):
            w[n] *= (9.0 / case["scale"] / dk) ** 0.5             # a key that matches its query scores about nine
        w["sink"] = w["sink"] * 3.0 + 2.0
        w["g"] *= 0.6
        if mix:
            w["vmix"] = torch.tensor(0.35)
    part, w64 = build_part("biased_attention", params, dtype, seed=dk, change=change)
    lengths = (290, 75, 1)
    xs = [x.to(dtype) for x in edge_inputs(lengths, hidden, case["window"], case["page"], seed=H)]
    m = dict(heads=H, kv_heads=G, dim=dk, vdim=dv, scale=case["scale"], softcap=case["cap"], v_mix=mix is not None)
    if case["rot"]:
        m["rot"] = dict(base=case["rot"][0], dims=case["rot"][1], scaling=scaling)
    first = None
    if mix:
        part, first = other_values(part, G * dv, hidden, dtype, mix != "plain", 18 if mix == "odd" else 16, seed=dv)

    def fn(x, window):
        f = None if first is None else first(x).view(-1, G, dv)
        return plain.rotated_attention(x.double(), w64, "m.", dict(m, mask=dict(size=window)), 2e-6, f)[0]
    want = [fn(x, case["window"]) for x in xs]
    check_edges(fn, case["window"], xs[0], want[0])
    whole, cutup = whole_then_portions(Bench(part, dtype, xs, want, page=case["page"]), lengths)
    limit = 3e-5 if dtype == torch.float32 else 0.06
    assert whole < limit and cutup < limit, (whole, cutup)


WHOLE_CASES = [dict(H=6, G=3, dk=40, dv=24, scale=0.25, window=37, page=16, mix="vec"),
               dict(H=3, G=1, dk=10, dv=6, scale=0.7, window=7, page=8, mix="odd"),
               dict(H=4, G=2, dk=128, dv=128, scale=0.09, window=100, page=32, mix="vec"),
               dict(H=2, G=1, dk=128, dv=128, scale=0.1, window=None, page=16, mix=None),
               dict(H=5, G=5, dk=12, dv=20, scale=0.5, window=64, page=16, mix="plain"),
               dict(H=4, G=1, dk=96, dv=48, scale=0.12, window=33, page=16, mix="vec"),
               dict(H=1, G=1, dk=300, dv=12, scale=0.06, window=16, page=16, mix="plain")]


@pytest.mark.parametrize("case", WHOLE_CASES, ids=lambda c: f"h{c['H']}g{c['G']}k{c['dk']}v{c['dv']}w{c['window']}")
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_normed_over_all_heads(case, dtype):
    from tiny_llm_infer_b200 import ops
    from tiny_llm_infer_b200.engine.runner import strict_float32
    strict_float32()
    H, G, dk, dv, hidden, mix = case["H"], case["G"], case["dk"], case["dv"], 96, case["mix"]
    params = dict(hidden_size=hidden, q_heads=H, kv_heads=G, key_dim=dk, value_dim=dv, scale=case["scale"], unit_norm_eps=3e-6,
                  qk_gains=True, norm_whole=True, window=case["window"], value_mix=None if mix is None else "mix")

    def change(w):
        for h in range(H):                                        # heads of different lengths: a norm per head would differ
            w["q"][h * dk:(h + 1) * dk] *= 0.6 + 0.3 * h
        tie(H, G, dk, hidden)(w)
        for n in ("q.norm", "k.norm"):
            w[n] = (w[n] * 0.3 + 0.7) * (10.0 / case["scale"] / dk) ** 0.5
        if mix:
            w["vmix"] = torch.tensor(0.6)
    part, w64 = build_part("biased_attention", params, dtype, seed=dk + 1, change=change)
    lengths = (290, 75, 1)
    xs = [x.to(dtype) for x in edge_inputs(lengths, hidden, case["window"], case["page"], seed=G)]
    m = dict(heads=H, kv_heads=G, dim=dk, vdim=dv, scale=case["scale"], v_mix=mix is not None)
    first = None
    if mix:
        part, first = other_values(part, G * dv, hidden, dtype, mix != "plain", 18 if mix == "odd" else 32, seed=dv)

    def fn(x, window):
        f = None if first is None else first(x).view(-1, G, dv)
        return plain.whole_normed_attention(x.double(), w64, "m.", dict(m, mask=dict(size=window)), 3e-6, f)[0]
    want = [fn(x, case["window"]) for x in xs]
    check_edges(fn, case["window"], xs[0], want[0])
    before = ops.tcgen05_calls
    whole, cutup = whole_then_portions(Bench(part, dtype, xs, want, page=case["page"]), lengths)
    ops.check_error_word(torch.device(DEV))
    if dtype == torch.bfloat16 and dk == dv == 128:
        assert ops.tcgen05_calls > before                         # the prompt kernel on the fifth-generation tensor cores
    limit = 3e-5 if dtype == torch.float32 else 0.06
    assert whole < limit and cutup < limit, (whole, cutup)


@pytest.mark.parametrize("kind,dk,dv,window", [("rotated", 64, 48, None), ("rotated", 96, 128, 700), ("whole", 128, 128, 900)])
def test_single_tokens_over_a_long_request(kind, dk, dv, window):
    """1200 tokens in one portion, then single tokens whose keys are dealt to several blocks and summed again: sink, cap
    and gate count once, and the window ends inside a block's run of keys."""
    from tiny_llm_infer_b200 import ops
    from tiny_llm_infer_b200.parts.spec import PartSpec
    H, G, hidden, dtype = 4, 1, 64, torch.bfloat16
    params = dict(hidden_size=hidden, q_heads=H, kv_heads=G, key_dim=dk, value_dim=dv, scale=0.1, unit_norm_eps=1e-6,
                  qk_gains=True, window=window, value_mix="first")
    if kind == "rotated":
        params.update(softcap=25.0, biases=True, output_bias=False, sink=True, learned_sink=True, output_gate=True,
                      gate_per_head=True, position=PartSpec("rotary_pairs", dict(head_dim=dk, theta=1e5, rotary_dim=8)))
    else:
        params["norm_whole"] = True

    def change(w):
        tie(H, G, dk, hidden)(w)
        for n in ("q.norm", "k.norm"):
            w[n] = (w[n] * 0.3 + 0.7) * (10.0 / 0.1 / dk) ** 0.5
        if "q.b" in w:
            w["q.b"] *= 0.5
            w["k.b"] *= 0.5
            w["sink"] += 4.0
    part, w64 = build_part("biased_attention", params, dtype, seed=dk + dv, change=change)
    L = 1230
    xs = [x.to(dtype) for x in edge_inputs((L,), hidden, window, 16, seed=5)]
    m = dict(heads=H, kv_heads=G, dim=dk, vdim=dv, scale=0.1, softcap=25.0, v_mix=True)
    if kind == "rotated":
        m["rot"] = dict(base=1e5, dims=8)
    fn = plain.rotated_attention if kind == "rotated" else plain.whole_normed_attention
    want = [fn(xs[0].double(), w64, "m.", dict(m, mask=dict(size=window)), 1e-6)[0]]
    bench = Bench(part, dtype, xs, want, page=16, slots=2)
    assert ops.biased_decode_splits(1, G, min(window or L, L)) > 1
    worst = bench.step([(0, 1, 0, 1200)])
    for p in range(1200, L):
        worst = max(worst, bench.step([(0, 1, p, 1)]))
    assert worst < 0.06, worst


# ----------------------------------------------------------------------------- the recurrence
DECAY_CASES = [dict(dk=24, dv=32, decay=(0.999, 0.6, 0.97)), dict(dk=10, dv=6, decay=(0.4, 0.998, 1.0, 0.9, 0.995)),
               dict(dk=64, dv=64, decay=(0.9985, 0.5)), dict(dk=128, dv=128, decay=(0.9, 0.999)), dict(dk=1, dv=3, decay=(0.999, 0.99)),
               dict(dk=8, dv=264, decay=(0.997,)), dict(dk=300, dv=5, decay=(0.2, 0.999)), dict(dk=40, dv=8, decay=(0.99, 0.0, 0.999))]


@pytest.mark.parametrize("case", DECAY_CASES, ids=lambda c: f"h{len(c['decay'])}k{c['dk']}v{c['dv']}")
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_recurrence_with_constant_decays(case, dtype):
    from tiny_llm_infer_b200.engine.runner import strict_float32
    strict_float32()
    H, dk, dv, hidden = len(case["decay"]), case["dk"], case["dv"], 72
    params = dict(hidden_size=hidden, heads=H, key_dim=dk, value_dim=dv, decays=case["decay"], norm_eps=2e-6)
    part, w64 = build_part("fixed_decay", params, dtype, seed=dk + dv)
    m = dict(heads=H, dim=dk, vdim=dv, decay=list(case["decay"]))
    whole, cutup = recurrence_run(part, w64, lambda x: plain.lightning(x, w64, "m.", m, 2e-6), dtype, hidden)
    limit = 3e-5 if dtype == torch.float32 else 0.06
    assert whole < limit and cutup < limit, (whole, cutup)


def test_recurrence_without_an_activation_and_with_a_scale():
    """The part's other options: q, k and v as projected, a scale on q, SiLU as the gate's activation."""
    H, dk, dv, hidden = 2, 16, 24, 40
    params = dict(hidden_size=hidden, heads=H, key_dim=dk, value_dim=dv, decays=(0.9, 0.99), norm_eps=1e-3, q_scale=0.05,
                  input_act=None, gate_act="silu")
    part, w = build_part("fixed_decay", params, torch.float32, seed=4)

    def fn(x):
        q, k, v = ((x @ w["m." + n].T).view(x.shape[0], H, -1) for n in "qkv")
        o = plain.fixed_decay_recurrence(q * 0.05, k, v, [0.9, 0.99]).reshape(x.shape[0], -1)
        return (plain.rms_unit(o, 1e-3) * w["m.norm"] * plain.silu(x @ w["m.g"].T)) @ w["m.o"].T
    x = torch.randn(50, hidden, generator=torch.Generator().manual_seed(1))
    assert Bench(part, torch.float32, [x], [fn(x.double())]).step([(0, 1, 0, 50)]) < 3e-5


@pytest.mark.parametrize("width,rows", [(72, 5), (4096, 3), (6, 9), (12288, 2), (130, 40)])
@pytest.mark.parametrize("gate_dtype", [torch.float32, torch.bfloat16])
def test_norm_over_all_heads_of_a_read_out(width, rows, gate_dtype):
    """Rows of one number alone, so that the mean is taken over the whole row; skipped rows come out as zeros."""
    from tiny_llm_infer_b200 import ops
    g = torch.Generator().manual_seed(width)
    dk, out_dtype = 2, torch.bfloat16
    proj = torch.randn(rows, 2 * dk + width, generator=g).to(out_dtype)
    proj = torch.cat([proj, torch.zeros(rows, -proj.shape[1] % 8, dtype=out_dtype)], 1).contiguous().to(DEV)
    gate = torch.randn(rows, width + 6, generator=g).to(gate_dtype).to(DEV)[:, 4:4 + width]
    weight = torch.rand(width, generator=g).to(DEV) + 0.5
    state = torch.zeros(rows, ops.linear_recurrence_state_floats("fixed_decay", 1, dk, width), device=DEV)
    slots = torch.arange(rows, dtype=torch.int32)
    slots[1] = -1
    out = ops.linear_recurrence(proj, "fixed_decay", None, torch.tensor([0.5], device=DEV), 1.0, gate, "sigmoid", weight, True,
                                1e-5, slots.to(DEV), None, state, 1, dk, width, 1.0, out_dtype, input_act="silu", norm_whole=True)
    p = plain.silu(proj.double())
    o = (p[:, :dk] * p[:, dk:2 * dk]).sum(1, keepdim=True) * p[:, 2 * dk:2 * dk + width]
    want = plain.rms_unit(o, 1e-5) * weight.double() * torch.sigmoid(gate.double())
    want[1] = 0
    assert (out.double() - want).abs().max() < 0.01 * want.abs().max()


# ----------------------------------------------------------------------------- ReLU units
def test_relu_in_the_products():
    """relu(g) u in the epilogues of the weight-streaming product (few rows), of the tcgen05 product (many), in the
    kernel of its own (between them and in float32) and in a mixture's grouped products."""
    from tiny_llm_infer_b200 import ops
    from tiny_llm_infer_b200.engine.runner import strict_float32
    from tiny_llm_infer_b200.parts.registry import lookup
    strict_float32()
    g = torch.Generator().manual_seed(19)
    gate, up, down = ((torch.randn(*s, generator=g) * 0.1).to(torch.bfloat16) for s in ((512, 256), (512, 256), (256, 512)))
    both = ops.interleave_gate_up(gate, up).contiguous().to(DEV)
    stacked = torch.cat([gate, up]).contiguous().to(DEV)
    for rows in (3, 40, 12000):
        x = torch.randn(rows, 256, generator=g).to(torch.bfloat16).to(DEV)
        want = torch.relu(x.double() @ gate.to(DEV).double().T) * (x.double() @ up.to(DEV).double().T)
        for wt, inter in ((both, True), (stacked, False)):
            got = ops.linear_swiglu(x, wt, torch.bfloat16, interleaved=inter, act="relu").double()
            assert (got - want).abs().max() < 0.02 * want.abs().max() and (got[want == 0] == 0).all()
    for dtype, inter, tol in ((torch.float32, 512, 1e-5), (torch.float32, 508, 1e-5), (torch.bfloat16, 508, 0.03)):
        part = lookup("feed_forward", "swiglu")(hidden_size=256, intermediate_size=inter, dtype=dtype, device=DEV, activation="relu",
                                                names=("gate", "up", "down"))
        w = dict(gate=gate[:inter].to(dtype), up=up[:inter].to(dtype), down=down[:, :inter].to(dtype).contiguous())
        part.load({k: v.to(DEV) for k, v in w.items()})
        x = torch.randn(21, 256, generator=g).to(dtype)
        want = plain.relu_unit(x.double(), {k: v.double() for k, v in w.items()}, "")
        assert (part.forward(x.to(DEV), None).double().cpu() - want).abs().max() < tol * want.abs().max()
    # a mixture of one expert is its expert: the grouped products, on mma.sync tiles, on tcgen05 and in float32
    for dtype, rows, tol in ((torch.bfloat16, 9, 0.03), (torch.bfloat16, 2100, 0.03), (torch.float32, 9, 1e-5)):
        part = lookup("feed_forward", "moe")(hidden_size=256, experts=1, top=1, expert_size=512, dtype=dtype, device=DEV,
                                             activation="relu", router_scores="softmax", weight_on="output")
        w = dict(gate=gate.to(dtype), up=up.to(dtype), down=down.to(dtype))
        part.load({"router": torch.zeros(1, 256, dtype=dtype, device=DEV), **{"e0." + k: v.to(DEV) for k, v in w.items()}})
        x = torch.randn(rows, 256, generator=g).to(dtype)
        want = plain.relu_unit(x.double(), {k: v.double() for k, v in w.items()}, "")
        assert (part.forward(x.to(DEV), None).double().cpu() - want).abs().max() < tol * want.abs().max()
    ops.check_error_word(torch.device(DEV))


# ----------------------------------------------------------------------------- whole models, every way of cutting
BF16_RMS = {"Z1": 0.07, "Z2": 0.075, "Z3": 0.04, "Z4": 0.04}


@pytest.fixture(scope="module", params=sorted(SOZAVIKS))
def case(request, tmp_path_factory):
    name = request.param
    tiny = SOZAVIKS[name]
    folder = make_folder(tiny, tmp_path_factory.mktemp(name))
    cfg, w = read_model(folder)
    reqs = requests_for(tiny)
    want = {rid: plain.forward(cfg, w, toks).numpy() for rid, toks in reqs.items()}
    tb = replay.TraceBuilder()
    replay.whole(tb, reqs)
    replay.tail_one_by_one(tb, reqs)
    replay.portions(tb, reqs)
    replay.mixed(tb, reqs, seed=11)
    return name, tiny, folder, cfg, w, want, tb, reqs


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_all_ways_of_cutting(case, dtype, tmp_path):
    name, tiny, folder, cfg, w, want, tb, reqs = case
    out = tmp_path / "out"
    run_tool(folder, dtype, out, tb, tiny["page_size"])
    errors, spread = relative_rows(out, tb, want, cfg["vocab"])
    assert set(errors) == {"w", "t", "p", "m"}
    summary = {k: (round(float(np.percentile(v, 50)), 6), round(float(v.max()), 6)) for k, v in errors.items()}
    between = {k: (round(float(np.percentile(v, 50)), 6), round(float(v.max()), 6)) for k, v in spread.items()}
    print(f"\n[{name} {dtype}] against plain (median, max) {summary}; between the ways (median, max) {between}")
    limit = 2e-5 if dtype == "float32" else BF16_RMS[name]
    assert max(v.max() for v in errors.values()) < limit, summary
    assert max(v.max() for v in spread.values()) < limit, between


def test_first_tokens_one_by_one_and_long_decoding(case, tmp_path):
    """One token at a time from an empty cache and empty states, beside a second request that decodes from the middle of
    a page; then the last 140 tokens of the longest request one by one (every window passes over decoded tokens alone);
    steps in which nothing is wanted lie between."""
    name, tiny, folder, cfg, w, want, _, reqs = case
    a, b = reqs["0"], reqs["1"]
    tb = replay.TraceBuilder()
    tb.step([("f1", b[:29])])
    for i in range(len(a)):
        extra = [("f1", b[29 + i:30 + i])] if 29 + i < len(b) else []
        tb.step([("f0", a[i:i + 1])] + extra)
    tb.step([], end=["f0", "f1"])
    long_one = max(reqs, key=lambda r: len(reqs[r]))
    replay.tail_one_by_one(tb, {long_one: reqs[long_one]}, tail=min(140, len(reqs[long_one]) - 3), tag="f")
    for n in (5, 8):
        for entry in tb.steps[n]["entries"]:
            entry["want"] = []
        tb.expect.pop(n)
    out = tmp_path / "out"
    run_tool(folder, "float32", out, tb, tiny["page_size"])
    errors, _ = relative_rows(out, tb, want, cfg["vocab"])
    assert errors["f"].max() < 2e-5, errors["f"].max()


# ----------------------------------------------------------------------------- generation through the entry point
def plain_greedy(cfg, w, prompt_ids, n):
    ids = list(prompt_ids)
    for _ in range(n):
        ids.append(int(plain.forward(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt_ids):]


def decisive_greedy(cfg, w, seeds_and_lengths, n):
    """Prompts whose greedy continuation of ``n`` tokens meets no near-tie of the last argmax."""
    prompts, wants = [], []
    for seed, length in seeds_and_lengths:
        for attempt in range(40):
            p = prompt(seed + 100 * attempt, length, cfg["vocab"])
            out = plain_greedy(cfg, w, p, n)
            logits = plain.forward(cfg, w, p + out)[len(p) - 1:-1]
            top2 = logits.topk(2, dim=-1).values
            if (top2[:, 0] - top2[:, 1]).min() > 1e-3 * logits.std():
                break
        prompts.append(p)
        wants.append(out)
    return prompts, wants


@pytest.mark.parametrize("name", ["Z1", "Z2"])
@pytest.mark.parametrize("budget,blocks", [(256, 64), (8, 64), (7, 14)])
def test_greedy_generation_equals_plain(name, budget, blocks, tmp_path):
    """Budgets down to seven tokens a step and a pool so small that requests are preempted and computed again
    (their states start from zero again), with decode steps replayed as CUDA graphs."""
    from tiny_llm_infer_b200 import LLM, SamplingParams
    tiny = SOZAVIKS[name]
    folder = make_folder(tiny, tmp_path)
    cfg, w = read_model(folder)
    prompts, want = decisive_greedy(cfg, w, [(0, 5), (1, 27), (2, 53), (3, 1)], 12)
    llm = LLM(str(folder), dtype="float32", max_model_len=128, num_kv_blocks=blocks, block_size=tiny["page_size"],
              max_num_batched_tokens=budget, max_num_seqs=3)
    outs = llm.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    assert [o.token_ids for o in outs] == want
    llm.cache.audit()
    assert all(v == blocks for v in llm.cache.free_pages().values())


def test_a_model_of_recurrent_layers_alone(tmp_path):
    """No attention: the cache manager has no group of pages at all and only the state slots."""
    from tiny_llm_infer_b200 import LLM, SamplingParams
    folder = make_folder(SOZAVIKS["Z4"], tmp_path)
    cfg, w = read_model(folder)
    prompts, want = decisive_greedy(cfg, w, [(7, 9), (8, 33), (9, 2), (10, 20)], 8)
    llm = LLM(str(folder), dtype="float32", max_model_len=96, num_kv_blocks=8, block_size=16, max_num_batched_tokens=16,
              max_num_seqs=2)
    assert not llm.cache.groups
    outs = llm.generate(prompts, SamplingParams(max_tokens=8, ignore_eos=True))
    assert [o.token_ids for o in outs] == want
    llm.cache.audit()


def test_long_decoding_in_bfloat16_through_graphs(tmp_path):
    """Sixty tokens each for three requests, decode steps replayed as CUDA graphs, bfloat16 kernels: every token
    is the plain implementation's choice given the same beginning, or within a near-tie of it."""
    from tiny_llm_infer_b200 import LLM, SamplingParams
    folder = make_folder(SOZAVIKS["Z3"], tmp_path)
    cfg, w = read_model(folder)
    prompts = [prompt(i, n, cfg["vocab"]) for i, n in enumerate((60, 9, 150))]
    llm = LLM(str(folder), dtype="bfloat16", max_model_len=256, num_kv_blocks=24, block_size=32,
              max_num_batched_tokens=64, max_num_seqs=3)
    outs = llm.generate(prompts, SamplingParams(max_tokens=60, ignore_eos=True))
    for p, o in zip(prompts, outs):
        ids = list(p) + list(o.token_ids)
        logits = plain.forward(cfg, w, ids[:-1]).numpy()
        near = [logits[len(p) - 1 + i][tok] >= logits[len(p) - 1 + i].max() - 0.15 * logits[len(p) - 1 + i].std()
                for i, tok in enumerate(o.token_ids)]
        assert sum(near) >= 0.9 * len(near), near


def test_command_line_writes_and_runs_a_model(tmp_path):
    """``bin/model_main``: a random Sozavik model from its config.json, greedy tokens equal to the plain implementation's
    in float32, and seeded sampling that repeats itself."""
    tiny = SOZAVIKS["Z2"]
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(tiny["cfg"].to_dict()))
    folder = tmp_path / "model"
    tool = [sys.executable, str(ROOT / "bin" / "model_main")]
    res = subprocess.run(tool + ["--write-random-model", str(folder), "--config", str(cfg_path), "--random-weights", "21",
                                 "--weight-std", "0.07"], capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    cfg, w = read_model(folder)
    prompts, want = decisive_greedy(cfg, w, [(40, 9), (41, 31)], 7)
    ids = [a for p in prompts for a in ("--prompt-ids", ",".join(map(str, p)))]
    common = tool + ["--infer", "--model", str(folder), "--max-seq-len", "128", "--max-new-tokens", "7"] + ids
    res = subprocess.run(common + ["--dtype", "float32"], capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    got = [[int(x) for x in line.split(",")] for line in res.stdout.strip().splitlines()[-2:]]
    assert got == want
    draws = []
    for _ in range(2):
        res = subprocess.run(common + ["--dtype", "bfloat16", "--temperature", "0.8", "--top-p", "0.9", "--seed", "5"],
                             capture_output=True, text=True, timeout=600)
        assert res.returncode == 0, res.stderr[-2000:]
        draws.append(res.stdout.strip().splitlines()[-2:])
    assert draws[0] == draws[1]
