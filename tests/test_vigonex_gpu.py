"""Vigonex on the GPU against the plain implementation (``plain_vigonex.py``).

Each mechanism alone, as the registered part or kernel with sizes of its own: the sinusoidal start; the kernel between
two sub-layers (update of the streams with gate and biases, weighted sum, norm, shift by a token), whole, in portions
and beside other requests; the attention with two maps per head over scrambled pages that hold other requests'
leftovers, with inputs shaped so that single keys far back, at page borders and next to the query stand out, in one or
in both maps; the delta rule with a removal rate per channel, whole, in portions down to one token, side by side and in
slots that are used again, with heads slow enough that the first tokens still show at the end; clamped experts, the
scaled router and the gated shared expert on every product kernel.  Then whole models through ``bin/trace_run`` in every
way of cutting, the first tokens one by one, long decoding, and greedy generation through the engine's entry point under
budgets and starved pools.

Tolerances, as a row's root-mean-square difference (its mean taken off) over the row's own spread: float32 2e-4
against the plain implementation and between the ways of cutting; bfloat16 three times what a B200 shows per
configuration."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import plain_vigonex as plain
import replay
from test_tetodra_gpu import (Bench, build_part, echo_inputs, make_ctx, read_model, relative_rows, run_tool, turn,
                              whole_then_portions)
from tiny_vigonex import VIGONEXES, make_folder, prompt, requests_for, slow_heads

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda:0"
F64 = torch.float64


# ----------------------------------------------------------------------------- the start
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,streams", [(96, 1), (37, 3), (2050, 2)])
def test_embedding_with_sinusoids(dtype, width, streams):
    """Positions up to many thousands of turns: float32 sines of the exact angle, not of a rounded one."""
    from tiny_llm_infer_b200.parts.embedding import SinusoidEmbedding
    g = torch.Generator().manual_seed(width)
    table = torch.randn(50, width, generator=g).to(dtype)
    part = SinusoidEmbedding(50, width, dtype, DEV, scale=1.7, name="e", streams=streams)
    part.load({"e": table.to(DEV)})
    ids = torch.tensor([3, 49, 0, -1, 7, 7], dtype=torch.int32)
    pos = [0, 1, 977, 5, 40001, 300007]

    class Ctx:
        positions = torch.tensor(pos, dtype=torch.int32, device=DEV)
    got = part.forward(ids.to(DEV), Ctx).view(6, streams, width).double().cpu()
    for r, (i, p) in enumerate(zip(ids.tolist(), pos)):
        if i < 0:
            assert got[r].abs().max() == 0
            continue
        col = torch.arange(width)
        ang = p * 10000.0 ** (-2.0 * (col // 2).double() / width)
        want = table[i].double() * 1.7 + torch.where(col % 2 == 0, torch.sin(ang), torch.cos(ang))
        for s in range(streams):
            assert (got[r, s] - want).abs().max() < 1e-6, (r, s)
    assert (plain.sinusoids(2, width, F64)[1] - (got[1, 0] - table[49].double() * 1.7)).abs().max() < 1e-6


# ----------------------------------------------------------------------------- between two sub-layers
def plain_between(x, S, w, delta, gate, shift):
    """x [T, S, D] float64 -> (streams after the update, h, shifted h)."""
    xs = x.transpose(0, 1)
    if delta is not None:
        y = delta + (w["db"] if w["db"] is not None else 0.0)
        if gate is not None:
            y = y * torch.sigmoid(gate + (w["gb"] if w["gb"] is not None else 0.0))
        xs = plain.write_streams(xs, w["mix"], w["out"], y)
    h = plain.rms_unit(plain.read_streams(xs, w["in"]), 3e-6) * w["gain"]
    return xs.transpose(0, 1), h, plain.token_shift(h, shift) if shift is not None else None


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,S,gated,bias", [(100, 2, True, True), (192, 3, True, False), (4104, 2, True, True), (37, 5, True, True),
                                                (64, 4, False, False), (128, 1, True, True), (88, 5, False, True), (9000, 4, True, True)])
def test_update_read_norm(dtype, width, S, gated, bias):
    """Without a shift: every number of streams, widths on and off the vector path, with and without gate and biases, an
    update or none, and chosen rows (which write nothing back)."""
    from tiny_llm_infer_b200 import ops
    g = torch.Generator().manual_seed(width + S)
    T = 11
    x = torch.randn(T, S * width, generator=g) * 3
    delta, gate = (torch.randn(T, width, generator=g) * 2).to(dtype), torch.randn(T, width, generator=g).to(dtype)
    w = {"in": torch.randn(S, generator=g), "out": torch.randn(S, generator=g), "mix": torch.randn(S, S, generator=g),
         "gain": torch.rand(width, generator=g) + 0.5, "db": torch.randn(width, generator=g) if bias else None,
         "gb": torch.randn(width, generator=g) if bias and gated else None}
    w64 = {k: v if v is None else v.double() for k, v in w.items()}
    d = {k: v if v is None else v.to(DEV) for k, v in w.items()}
    X = x.double().view(T, S, width)
    new, h, _ = plain_between(X, S, w64, delta.double(), gate.double() if gated else None, None)
    args = dict(w_in=d["in"], delta=delta.to(DEV), mix=d["mix"], w_out=d["out"], delta_bias=d["db"],
                gate=gate.to(DEV) if gated else None, gate_bias=d["gb"])
    xd = x.to(DEV)
    got_x, got_h, none = ops.stream_read(xd, S, d["gain"], 3e-6, dtype, **args)
    tol = 3e-5 if dtype == torch.float32 else 0.03
    assert none is None and torch.equal(xd.cpu(), x)
    assert (got_x.double().cpu().view(T, S, width) - new).abs().max() < 3e-5 * new.abs().max()     # float32 whatever the mode
    assert (got_h.double().cpu() - h).abs().max() < tol * max(1.0, float(h.abs().max()) / 4)
    rows = torch.tensor([7, 0, -1, 10], dtype=torch.int32, device=DEV)
    none, chosen, _ = ops.stream_read(xd, S, d["gain"], 3e-6, dtype, rows=rows, **args)
    assert none is None and chosen[2].abs().max() == 0 and torch.equal(chosen[[0, 1, 3]], got_h[[7, 0, 10]])
    # no update: the plain sum of the streams
    same, got_h, _ = ops.stream_read(xd, S, d["gain"], 3e-6, dtype)
    want = plain.rms_unit(X.sum(1), 3e-6) * w64["gain"]
    assert same is xd and (got_h.double().cpu() - want).abs().max() < tol
    empty = ops.stream_read(xd, S, d["gain"], 3e-6, dtype, rows=rows[:0], **args)[1]
    assert tuple(empty.shape) == (0, width)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,S", [(72, 3), (37, 2), (640, 1), (40, 5)])
def test_shift_by_a_token_in_portions(dtype, width, S):
    """The shifted input of a request of 150 tokens, whole and in portions down to one token beside other requests and in
    a slot that was used before; the streams' update goes along.  Rows of h equal whichever way, bit for bit."""
    from tiny_llm_infer_b200 import ops
    g = torch.Generator().manual_seed(width)
    lengths = (150, 61, 1)
    w = {"in": torch.randn(S, generator=g), "out": torch.randn(S, generator=g), "mix": torch.randn(S, S, generator=g),
         "gain": torch.rand(width, generator=g) + 0.5, "db": torch.randn(width, generator=g), "gb": torch.randn(width, generator=g)}
    shift = torch.rand(width, generator=g) * 1.5 - 0.25
    w64 = {k: v.double() for k, v in w.items()}
    d = {k: v.to(DEV) for k, v in w.items()}
    reqs = [(torch.randn(L, S * width, generator=g) * 3, (torch.randn(L, width, generator=g) * 2).to(dtype),
             torch.randn(L, width, generator=g).to(dtype)) for L in lengths]
    want = [plain_between(x.double().view(-1, S, width), S, w64, dl.double(), gt.double(), None)[1] for x, dl, gt in reqs]
    tail = torch.zeros(4, width, device=DEV)
    first = {}

    def step(rows):
        """rows: (request, slot, first position, count)."""
        ctx = make_ctx([(slot, p0, n) for _, slot, p0, n in rows])
        cat = [torch.cat([reqs[r][k][p0:p0 + n] for r, _, p0, n in rows]).to(DEV) for k in range(3)]
        _, h, s = ops.stream_read(cat[0], S, d["gain"], 3e-6, dtype, w_in=d["in"], delta=cat[1], mix=d["mix"], w_out=d["out"],
                                  delta_bias=d["db"], gate=cat[2], gate_bias=d["gb"], shift=shift.to(DEV), tail=tail,
                                  token_slot=ctx.token_slot, seg_info=ctx.seg_info, single_tokens=ctx.decode_only)
        at = 0
        for r, _, p0, n in rows:
            for i in range(n):
                p = p0 + i
                hp, sp = h[at].clone(), s[at].clone()
                if (r, p) in first:
                    assert torch.equal(first[(r, p)][0], hp) and torch.equal(first[(r, p)][1], sp), (r, p)
                first[(r, p)] = (hp, sp)
                before = first[(r, p - 1)][0].double() if p else torch.zeros(width, dtype=F64, device=DEV)
                expect = hp.double() + (before - hp.double()) * shift.double().to(DEV)
                scale = max(1.0, float(expect.abs().max()))
                assert (sp.double() - expect).abs().max() < (1e-6 if dtype == torch.float32 else 0.01) * scale, (r, p)
                tol = 3e-5 if dtype == torch.float32 else 0.02
                assert (hp.double().cpu() - want[r][p]).abs().max() < tol * max(1.0, float(want[r][p].abs().max())), (r, p)
                at += 1
    step([(0, 2, 0, lengths[0]), (1, 0, 0, lengths[1]), (2, 3, 0, 1)])
    tail[2].zero_()
    tail[0].zero_()
    at0 = at1 = k = 0
    sizes = [1, 1, 2, 1, 3, 2, 17, 2, 1, 16, 33, 1, 64, 5]
    while at0 < lengths[0]:
        n0 = min(sizes[k % len(sizes)], lengths[0] - at0)
        rows = [(0, 0, at0, n0)]
        if at1 < lengths[1] and k % 3 != 1:
            n1 = min(sizes[(k + 5) % len(sizes)], lengths[1] - at1)
            rows.append((1, 2, at1, n1))
            at1 += n1
        step(rows)
        at0 += n0
        k += 1


@pytest.mark.parametrize("width,S,T", [(64, 2, 5000), (64, 5, 5000), (4096, 2, 1500)])
def test_shift_over_a_long_portion(width, S, T):
    """So many rows that a block walks a run of them: the row before a run is computed once more."""
    from tiny_llm_infer_b200 import ops
    torch.manual_seed(T)
    x = torch.randn(T, S * width, device=DEV)
    delta = torch.randn(T, width, device=DEV).to(torch.bfloat16)
    gate = torch.randn(T, width, device=DEV).to(torch.bfloat16)
    w = [torch.randn(S, device=DEV), torch.randn(S, device=DEV), torch.randn(S, S, device=DEV)]
    gain, shift = torch.rand(width, device=DEV) + 0.5, torch.rand(width, device=DEV)
    a, b = T // 3, T - T // 3 - 1                                   # two requests and one of a single token
    ctx = make_ctx([(1, 40, a), (3, 0, 1), (0, 7, b)])
    tail = torch.randn(4, width, device=DEV)
    before = tail.clone()
    _, h, s = ops.stream_read(x, S, gain, 1e-5, torch.bfloat16, w_in=w[0], delta=delta, mix=w[2], w_out=w[1], gate=gate, shift=shift,
                              tail=tail, token_slot=ctx.token_slot, seg_info=ctx.seg_info)
    y = delta.double() * torch.sigmoid(gate.double())
    X = torch.einsum("tsd,su->tud", x.double().view(T, S, width), w[2].double()) + w[1].double().view(1, S, 1) * y.unsqueeze(1)
    u = torch.einsum("tsd,s->td", X, w[0].double())
    want = plain.rms_unit(u, 1e-5) * gain.double()
    assert (h.double() - want).abs().max() < 0.02 * want.abs().max()
    prev = torch.cat([h[:1], h[:-1]]).double()
    prev[0], prev[a], prev[a + 1] = before[1].double(), before[3].double(), before[0].double()
    expect = h.double() + (prev - h.double()) * shift.double()
    assert (s.double() - expect).abs().max() < 0.01 * expect.abs().max()
    for slot, last in ((1, a - 1), (3, a), (0, T - 1)):
        assert torch.equal(tail[slot], h[last].float())
    assert torch.equal(tail[2], before[2])


# ----------------------------------------------------------------------------- attention with two maps per head
MAPS_CASES = [dict(H=6, G=2, dk=24, dv=40, scale=0.3, diff=0.3, cap=9.0, temp=(0.4, 16), page=16),
              dict(H=1, G=1, dk=10, dv=6, scale=0.5, diff=0.2, cap=4.0, temp=(0.8, 7), page=8),
              dict(H=4, G=1, dk=6, dv=22, scale=0.6, diff=0.45, cap=None, temp=None, page=8),
              dict(H=4, G=2, dk=64, dv=128, scale=0.1, diff=0.8, cap=20.0, temp=(0.35, 64), page=32),
              dict(H=8, G=1, dk=128, dv=64, scale=0.08, diff=0.35, cap=40.0, temp=(0.5, 100), page=32),
              dict(H=20, G=1, dk=32, dv=32, scale=0.2, diff=0.5, cap=None, temp=(0.2, 1000), page=16),
              dict(H=3, G=3, dk=16, dv=200, scale=0.4, diff=0.6, cap=12.0, temp=(0.3, 33), page=16),
              dict(H=2, G=2, dk=128, dv=128, scale=0.07, diff=0.4, cap=None, temp=(0.1, 1), page=16)]


def tie_maps(H, G, dk, hidden):
    """Keys that echo the first query head of their group (``echo_inputs``): in both maps for even key heads, in the
    second map only for odd ones (the first then has no key that stands out)."""
    R = turn(hidden)

    def change(w):
        for kv in range(G):
            first = kv * (H // G)
            for m in (0, 1) if kv % 2 == 0 else (1,):
                at, src = (2 * kv + m) * dk, (2 * first + m) * dk
                w["k"][at:at + dk] = w["q"][src:src + dk] @ R
                w["k.b"][at:at + dk] = w["q.b"][src:src + dk] * 0.3
        w["q.b"] *= 0.3
        for n in ("lq1", "lk1", "lq2", "lk2"):
            w[n] *= 0.3
    return change


def maps_part(case, dtype, hidden, defer=True):
    params = dict(hidden_size=hidden, q_heads=case["H"], kv_heads=case["G"], key_dim=case["dk"], value_dim=case["dv"],
                  scale=case["scale"], softcap=case["cap"], q_temperature=case["temp"], biases=True, defer_output_bias=defer,
                  differential=(case["diff"], 2e-6))
    part, w64 = build_part("biased_attention", params, dtype, seed=case["dk"] + case["dv"],
                           change=tie_maps(case["H"], case["G"], case["dk"], hidden), stds={"q": 0.2, "k": 0.2})
    m = dict(heads=case["H"], kv_heads=case["G"], dim=case["dk"], vdim=case["dv"], scale=case["scale"], softcap=case["cap"],
             diff=case["diff"], q_temp=None if case["temp"] is None else dict(coef=case["temp"][0], every=case["temp"][1]))
    return part, w64, m


@pytest.mark.parametrize("case", MAPS_CASES, ids=lambda c: f"h{c['H']}g{c['G']}k{c['dk']}v{c['dv']}")
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_with_two_maps(case, dtype):
    from tiny_llm_infer_b200.engine.runner import strict_float32
    strict_float32()
    hidden, defer = 104, case["H"] != 4
    part, w64, m = maps_part(case, dtype, hidden, defer)
    lengths = (290, 75, 1)
    xs = [x.to(dtype) for x in echo_inputs(lengths, hidden, case["page"], seed=case["H"])]
    want = [plain.differential_attention(x.double(), w64, "m.", m, 2e-6) for x in xs]
    cut = plain.differential_attention(xs[0][40:].double(), w64, "m.", m, 2e-6)
    assert (cut[-1] - want[0][-1]).abs().max() > 0.01 * want[0].abs().max()
    if defer:                                                   # the block's kernel adds it: the part leaves it out
        assert part.deferred_bias is not None and part.out_bias is None
        want = [x - w64["m.o.b"] for x in want]
    whole, cutup = whole_then_portions(Bench(part, dtype, xs, want, page=case["page"]), lengths)
    limit = 3e-5 if dtype == torch.float32 else 0.06
    assert whole < limit and cutup < limit, (whole, cutup)


@pytest.mark.parametrize("case", [MAPS_CASES[0], MAPS_CASES[3], MAPS_CASES[4]], ids=lambda c: f"h{c['H']}g{c['G']}k{c['dk']}v{c['dv']}")
def test_two_maps_over_a_long_request_with_shared_out_keys(case):
    """Single tokens at the end of 1200: the keys of a row are dealt to several blocks, whose partial sums of both maps
    meet in the combining kernel; prompt portions of several blocks of rows before them."""
    from tiny_llm_infer_b200 import ops
    hidden, L, dtype = 104, 1200, torch.bfloat16
    part, w64, m = maps_part(case, dtype, hidden)
    xs = [x.to(dtype) for x in echo_inputs((L, 3), hidden, case["page"], seed=case["H"] + 50)]
    want = [plain.differential_attention(x.double(), w64, "m.", m, 2e-6) - w64["m.o.b"] for x in xs]
    assert ops.biased_decode_splits(1, case["G"], L) > 1
    bench = Bench(part, dtype, xs, want, page=case["page"])
    worst = bench.step([(0, 1, 0, 700), (1, 2, 0, 3)])
    worst = max(worst, bench.step([(0, 1, 700, 470)]))
    for p in range(1170, L):
        worst = max(worst, bench.step([(0, 1, p, 1)]))
    assert worst < 0.06, worst


# ----------------------------------------------------------------------------- the delta rule with a removal rate per channel
ERASE_CASES = [dict(H=4, d=16, rank=8), dict(H=3, d=10, rank=5), dict(H=2, d=128, rank=24), dict(H=1, d=72, rank=16),
               dict(H=5, d=64, rank=8), dict(H=2, d=200, rank=3), dict(H=1, d=264, rank=8), dict(H=7, d=1, rank=2),
               dict(H=6, d=32, dv=56, rank=8), dict(H=2, d=20, dv=6, rank=4),
               dict(H=10, d=128, rank=8), dict(H=21, d=60, rank=8), dict(H=8, d=200, rank=4)]     # two columns per thread


@pytest.mark.parametrize("case", ERASE_CASES, ids=lambda c: f"h{c['H']}d{c['d']}v{c.get('dv', c['d'])}r{c['rank']}")
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_delta_rule_with_removal_per_channel(case, dtype):
    """Every second head forgets a thousandth a token and overwrites about a hundredth, so that the first tokens still
    show after hundreds; keys from a tenth to several units long (only their direction removes)."""
    from tiny_llm_infer_b200.engine.runner import strict_float32
    strict_float32()
    hidden, H, d, dv = 80, case["H"], case["d"], case.get("dv", case["d"])
    params = dict(hidden_size=hidden, heads=H, key_dim=d, value_dim=dv, decay_rank=case["rank"], norm_eps=1e-5)

    def change(w):
        w["w0"], w["a.b"] = slow_heads(w["w0"], w["a.b"], H)
        w["k"] = w["k"] * torch.linspace(0.2, 3.0, H).repeat_interleave(d).unsqueeze(1)
    part, w64 = build_part("erase_delta", params, dtype, seed=d + dv, change=change,
                           stds={n: 0.12 for n in ("r", "k", "v", "g", "a", "w1")})

    def fn(x):
        if dv == d:
            return plain.general_delta(x, w64, "m.", dict(heads=H, dim=d), 1e-5)
        # the same equations with values of another width
        T = x.shape[0]
        r, k, v = ((x @ w64["m." + n].T).view(T, H, -1) for n in "rkv")
        z = torch.tanh(x @ w64["m.w1"].T) @ w64["m.w2"].T + w64["m.w0"]
        w = torch.exp(-torch.exp(torch.tensor(-0.5, dtype=F64)) * torch.sigmoid(z)).view(T, H, d)
        a = torch.sigmoid(x @ w64["m.a"].T + w64["m.a.b"]).view(T, H, d)
        u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        S, out = torch.zeros(H, d, dv, dtype=F64), []
        for t in range(T):
            read = torch.einsum("hk,hkv->hv", u[t], S)
            S = w[t].unsqueeze(-1) * S - torch.einsum("hk,hv->hkv", a[t] * u[t], read) + torch.einsum("hk,hv->hkv", k[t], v[t])
            out.append(torch.einsum("hkv,hk->hv", S, r[t]))
        o = plain.rms_unit(torch.stack(out), 1e-5).reshape(T, H * dv) * w64["m.norm"] * torch.sigmoid(x @ w64["m.g"].T)
        return o @ w64["m.o"].T
    lengths = (230, 61, 1)
    g = torch.Generator().manual_seed(5)
    xs = [torch.randn(L, hidden, generator=g).to(dtype) for L in lengths]
    want = [fn(x.double()) for x in xs]
    if d > 1:
        short = fn(xs[0][30:].double())
        assert (short[-1] - want[0][-1]).abs().max() > 1e-3 * want[0].abs().max()
    whole, cutup = whole_then_portions(Bench(part, dtype, xs, want), lengths)
    limit = 3e-5 if dtype == torch.float32 else 0.06
    if d == 1:                     # a head of one number is normed to its sign: a read-out near zero may fall either way
        limit = 1e-3 if dtype == torch.float32 else 2.0
    assert whole < limit and cutup < limit, (whole, cutup)


@pytest.mark.parametrize("dk,dv", [(64, 96), (128, 64), (250, 40)])
@pytest.mark.parametrize("mode", ["delta", "channel_decay", "log_gates", "state_space", "erase", "fixed_decay"])
def test_scan_with_two_columns_per_thread_changes_nothing(mode, dk, dv):
    """Every recurrence of the scan kernel: portions of 48 tokens (two columns per thread at these sizes) against the same
    tokens in portions of 8 (one), bit for bit, states included."""
    from tiny_llm_infer_b200 import ops
    H, slots, L = 3552 // (3 * dv) + 4, 3, 48
    torch.manual_seed(dk)
    if mode == "state_space":
        width, words = 2 * H * dv + 2 * H * dk + H, ops.state_space_state_floats(H, H, dk, dv, 1)
    elif mode == "erase":
        width, words = 3 * H * dk + 2 * H * dv, ops.delta_rule_state_floats(H, H, dk, dv, 1)
    elif mode == "delta":
        width, words = 2 * H * dk + H * dv + H, ops.delta_rule_state_floats(H, H, dk, dv, 1)
    else:
        width, words = H * (2 * dk + dv), ops.linear_recurrence_state_floats(mode, H, dk, dv)
    proj = torch.randn(slots, L, -(-width // 8) * 8, device=DEV) * 0.3
    z = torch.randn(slots, L, 2 * H if mode == "log_gates" else H * dk, device=DEV)
    gate = torch.randn(slots, L, H * dv, device=DEV)
    zb, ab, rate = torch.randn(z.shape[2], device=DEV), torch.randn(H * dk, device=DEV), torch.rand(H, device=DEV)
    w1, wh, hb = torch.ones(dv, device=DEV), torch.ones(H * dv, device=DEV), torch.randn(H, device=DEV)
    conv = torch.ones(2 * H * dk + H * dv, 1, device=DEV)

    def run(step):
        state = torch.zeros(slots, words, device=DEV)
        outs = []
        for p0 in range(0, L, step):
            cut = [t[:, p0:p0 + step].reshape(slots * step, -1).contiguous() for t in (proj, z, gate)]
            ctx = make_ctx([(i, p0, step) for i in range(slots)])
            common = (ctx.token_slot, ctx.seg_info, state)
            f32 = torch.float32
            if mode == "erase":
                o = ops.erase_delta_rule(cut[0], 2 * H * dk + 2 * H * dv, cut[1], zb, ab, 0.6, cut[2], "sigmoid", wh, True, 1e-6, *common,
                                         H, dk, dv, 1e-6, f32)
            elif mode == "delta":
                o = ops.delta_rule(cut[0], conv, 1, cut[1], zb, rate, cut[2], w1, 1e-6, *common, H, H, dk, dv, 0.1, 1e-6, f32)
            elif mode == "state_space":
                o = ops.state_space(cut[0], conv, None, 1, hb, rate, hb, wh, 1e-6, 1, *common, H, H, dk, dv, f32)
            elif mode == "fixed_decay":
                o = ops.linear_recurrence(cut[0], mode, None, rate, 1.0, cut[2], "sigmoid", wh, True, 1e-6, *common, H, dk, dv, 0.1, f32,
                                          input_act="silu", norm_whole=True)
            else:
                o = ops.linear_recurrence(cut[0], mode, cut[1], zb, 8.0, cut[2], "silu", w1, False, 1e-6, *common, H, dk, dv, 0.1, f32)
            outs.append(o.view(slots, step, -1))
        return torch.cat(outs, dim=1), state
    (long, s1), (short, s2) = run(L), run(8)
    assert torch.isfinite(long).all() and long.abs().max() > 0
    assert torch.equal(long, short) and torch.equal(s1, s2)


# ----------------------------------------------------------------------------- experts
MIXTURE_CASES = [dict(hidden=96, E=6, top=2, ff=48, limit=0.8, scale=1.5, shared=64, slimit=1.2, rows=37),
                 dict(hidden=101, E=5, top=3, ff=30, limit=1.1, scale=0.7, shared=22, slimit=0.6, rows=9),
                 dict(hidden=128, E=9, top=4, ff=64, limit=2.0, scale=1.0, shared=136, slimit=0.5, rows=1500),
                 dict(hidden=64, E=4, top=1, ff=12, limit=0.7, scale=2.0, shared=None, slimit=None, rows=3),
                 dict(hidden=256, E=8, top=8, ff=40, limit=1.0, scale=0.3, shared=512, slimit=0.9, rows=2100)]


@pytest.mark.parametrize("case", MIXTURE_CASES, ids=lambda c: f"h{c['hidden']}e{c['E']}t{c['top']}r{c['rows']}")
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_mixture_of_clamped_experts(case, dtype):
    """The registered part against the plain mixture: few rows (tiles of 64 on mma.sync, or one thread per output), many
    (the grouped tcgen05 product), gates and ups that reach their limits on both sides, every expert chosen or one."""
    from tiny_llm_infer_b200 import ops
    from tiny_llm_infer_b200.engine.runner import strict_float32
    from tiny_llm_infer_b200.parts.registry import lookup
    from tiny_llm_infer_b200.parts.spec import PartSpec
    strict_float32()
    hidden, names = case["hidden"], ("gate", "up", "down")
    shared = None
    if case["shared"]:
        shared = PartSpec("swiglu", dict(hidden_size=hidden, intermediate_size=case["shared"], activation="clamped_swish",
                                         act_consts=(case["slimit"], 1.702), names=names), "shared.")
    params = dict(hidden_size=hidden, experts=case["E"], top=case["top"], expert_size=case["ff"], activation="clamped_swish",
                  act_consts=(case["limit"], 1.702), router_scores="softmax_all", router_scale=case["scale"], weight_on="output",
                  shared=shared, shared_gate="sg" if shared else None, names=names)
    cls = lookup("feed_forward", "moe")
    g = torch.Generator().manual_seed(hidden + case["rows"])
    w = {}
    for name, spec in cls.param_specs(**params).items():
        std = 3.0 / hidden ** 0.5 if name == "router" else (1.5 / hidden ** 0.5 if not name.endswith("down") else 0.25)
        w[name] = (torch.randn(spec.shape, generator=g) * std).to(dtype)
    part = cls(dtype=dtype, device=DEV, **params)
    part.load({k: v.to(DEV) for k, v in w.items()})
    w64 = {"m." + k: v.double() for k, v in w.items()}
    x = torch.randn(case["rows"], hidden, generator=g).to(dtype)
    mlp = dict(expert=dict(limit=case["limit"]), router=dict(experts=case["E"], top=case["top"], scale=case["scale"]),
               shared=dict(limit=case["slimit"]) if case["shared"] else None)
    z = x.double() @ w64["m.e0.gate"].T
    assert (z > case["limit"]).any() and (z < -case["limit"]).any()
    want = plain.mixture(x.double(), w64, "m.", mlp)
    sure = plain.router_margin(x.double(), w64["m.router"], case["top"]) > (1e-4 if dtype == torch.float32 else 0.05)
    assert sure.float().mean() > 0.5
    got = part.forward(x.to(DEV), None).double().cpu()
    ops.check_error_word(torch.device(DEV))
    err = ((got - want)[sure].abs().max() / want.abs().max()).item()
    assert err < (3e-5 if dtype == torch.float32 else 0.03), err


def test_clamped_swish_and_tanh_in_the_products():
    """g sigmoid(slope g) (u + 1) with its bounds, and tanh, in the epilogues of the weight-streaming product (few rows),
    of the tcgen05 product (many) and in the kernels of their own (between them); another slope than the design's."""
    from tiny_llm_infer_b200 import ops
    g = torch.Generator().manual_seed(9)
    gate, up = ((torch.randn(512, 256, generator=g) * 0.1).to(torch.bfloat16) for _ in range(2))
    both = ops.interleave_gate_up(gate, up).contiguous().to(DEV)
    stacked = torch.cat([gate, up]).contiguous().to(DEV)
    eye = torch.eye(512, dtype=F64)
    for rows in (3, 40, 12000):
        x = torch.randn(rows, 256, generator=g).to(torch.bfloat16)
        zg, zu = (x.to(DEV).double() @ m.to(DEV).double().T for m in (gate, up))
        cg, cu = torch.clamp(zg, max=0.9), torch.clamp(zu, -0.9, 0.9)
        want = cg * torch.sigmoid(2.5 * cg) * (cu + 1.0)
        for wt, inter in ((both, True), (stacked, False)):
            got = ops.linear_swiglu(x.to(DEV), wt, torch.bfloat16, interleaved=inter, act="clamped_swish", consts=(0.9, 2.5)).double()
            assert (got - want).abs().max() < 0.02 * want.abs().max()
        got = ops.linear_act(x.to(DEV), stacked, "tanh", torch.bfloat16).double()
        assert (got - torch.tanh(torch.cat([zg, zu], dim=1))).abs().max() < 0.01
    small = plain.clamped_expert(x[:4].double(), gate.double(), up.double(), eye, 0.9)
    assert (small - torch.clamp(zg[:4], max=0.9).cpu() * torch.sigmoid(1.702 * torch.clamp(zg[:4], max=0.9).cpu())
            * (torch.clamp(zu[:4], -0.9, 0.9).cpu() + 1)).abs().max() < 1e-9
    with pytest.raises(ops.KernelError, match="constants"):
        ops.linear_swiglu(x[:3].to(DEV), both, torch.bfloat16, interleaved=True, act="clamped_swish")
    ops.check_error_word(torch.device(DEV))


@pytest.mark.parametrize("E,top,scale", [(6, 2, 1.5), (257, 8, 0.4), (3, 3, 1.0)])
def test_router_with_a_scale_and_more_columns(E, top, scale):
    from tiny_llm_infer_b200 import ops
    g = torch.Generator().manual_seed(E)
    z = torch.randn(500, E + 1, generator=g) * 2.0                    # one more column behind the logits, larger than all
    z[:, E] = 50.0
    chosen, weights = plain.route(z[:, :E].double(), torch.eye(E, dtype=F64), top, scale)
    ids, wts = ops.moe_route_grouped(z.to(DEV), top, "softmax", scale=scale, experts=E)
    sure = plain.router_margin(z[:, :E].double(), torch.eye(E, dtype=F64), top) > 1e-4
    got, want = ids.cpu().long().sort(-1), chosen.sort(-1)
    assert sure.float().mean() > 0.9 and torch.equal(got.values[sure], want.values[sure])
    gw, ww = torch.gather(wts.cpu().double(), 1, got.indices), torch.gather(weights, 1, want.indices)
    assert (gw[sure] - ww[sure]).abs().max() < 1e-6


# ----------------------------------------------------------------------------- whole models, every way of cutting
BF16_RMS = {"G1": 0.16, "G2": 0.05, "G3": 0.06, "G4": 0.05}


@pytest.fixture(scope="module", params=sorted(VIGONEXES))
def case(request, tmp_path_factory):
    name = request.param
    tiny = VIGONEXES[name]
    folder = make_folder(tiny, tmp_path_factory.mktemp(name))
    cfg, w = read_model(folder)
    reqs = {rid: plain.decisive_tokens(cfg, w, toks, seed=int(rid)) for rid, toks in requests_for(tiny).items()}
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
    limit = 2e-4 if dtype == "float32" else BF16_RMS[name]
    assert max(v.max() for v in errors.values()) < limit, summary
    assert max(v.max() for v in spread.values()) < limit, between


def test_first_tokens_one_by_one_and_long_decoding(case, tmp_path):
    """One token at a time from an empty cache and empty states (no token before the first, the state's first writes),
    beside a second request that decodes from the middle of a page; then the last 140 tokens of the longest request one
    by one; steps in which nothing is wanted lie between."""
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
    for n in (5, 8):                                             # unwanted rows among the portions and the single tokens
        for entry in tb.steps[n]["entries"]:
            entry["want"] = []
        tb.expect.pop(n)
    out = tmp_path / "out"
    run_tool(folder, "float32", out, tb, tiny["page_size"])
    errors, _ = relative_rows(out, tb, want, cfg["vocab"])
    assert errors["f"].max() < 2e-4, errors["f"].max()


# ----------------------------------------------------------------------------- generation through the entry point
def plain_greedy(cfg, w, prompt_ids, n):
    ids = list(prompt_ids)
    for _ in range(n):
        ids.append(int(plain.forward(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt_ids):]


def decisive_greedy(cfg, w, seeds_and_lengths, n):
    """Prompts whose greedy continuation of ``n`` tokens meets no near-tie of a router or of the last argmax."""
    prompts, wants = [], []
    for seed, length in seeds_and_lengths:
        for attempt in range(40):
            p = plain.decisive_tokens(cfg, w, prompt(seed + 100 * attempt, length, cfg["vocab"]), seed=seed, threshold=3e-3)
            out = plain_greedy(cfg, w, p, n)
            gaps = []
            logits = plain.forward(cfg, w, p + out, gaps_out=gaps)[len(p) - 1:-1]
            top2 = logits.topk(2, dim=-1).values
            if (top2[:, 0] - top2[:, 1]).min() > 1e-3 * logits.std() and (not gaps or torch.stack(gaps).min() > 1e-3):
                break
        prompts.append(p)
        wants.append(out)
    return prompts, wants


@pytest.mark.parametrize("name", ["G1", "G2"])
@pytest.mark.parametrize("budget,blocks", [(256, 64), (8, 64), (7, 14)])
def test_greedy_generation_equals_plain(name, budget, blocks, tmp_path):
    """Budgets down to seven tokens a step and a pool so small that requests are preempted and computed again
    (their states start from zero again), with decode steps replayed as CUDA graphs."""
    from tiny_llm_infer_b200 import LLM, SamplingParams
    tiny = VIGONEXES[name]
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
    """No attention anywhere: no pages, only states (the shift's and the delta rule's)."""
    from tiny_llm_infer_b200 import LLM, SamplingParams
    tiny = VIGONEXES["G4"]
    folder = make_folder(tiny, tmp_path)
    cfg, w = read_model(folder)
    prompts, want = decisive_greedy(cfg, w, [(7, 9), (8, 33), (9, 2), (10, 20)], 8)
    llm = LLM(str(folder), dtype="float32", max_model_len=96, num_kv_blocks=32, block_size=16, max_num_batched_tokens=16,
              max_num_seqs=2)
    outs = llm.generate(prompts, SamplingParams(max_tokens=8, ignore_eos=True))
    assert [o.token_ids for o in outs] == want


def test_long_decoding_in_bfloat16_through_graphs(tmp_path):
    """Sixty tokens each for three requests, decode steps replayed as CUDA graphs, bfloat16 kernels: every token
    is the plain implementation's choice given the same beginning, or within a near-tie of it."""
    from tiny_llm_infer_b200 import LLM, SamplingParams
    tiny = VIGONEXES["G3"]
    folder = make_folder(tiny, tmp_path)
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
        assert sum(near) >= 0.85 * len(near), near


def test_command_line_writes_and_runs_a_model(tmp_path):
    """``bin/model_main``: a random Vigonex model from its config.json, greedy tokens equal to the plain implementation's
    in float32, and seeded sampling that repeats itself."""
    tiny = VIGONEXES["G2"]
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
