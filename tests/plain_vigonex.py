"""Vigonex, plainly: whole sequences, no cache, no batching, float64 unless told otherwise; one
function per mechanism.  It shares no code with the engine and is what the engine is compared with.

``weights`` maps tensor names to torch tensors (any float type), ``cfg`` is the dictionary of
config.json.  Notation: T tokens, D the model width, rows are tokens.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

UNIT_EPS = 1e-6


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def sinusoids(T: int, width: int, dtype) -> torch.Tensor:
    """[T, width]: column 2i is sin(p f_i), column 2i + 1 cos(p f_i), f_i = 10000^(-2i / width)."""
    out = torch.zeros(T, width, dtype=dtype)
    p = torch.arange(T, dtype=torch.float64)
    for c in range(width):
        ang = p * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = (torch.sin(ang) if c % 2 == 0 else torch.cos(ang)).to(dtype)
    return out


# ---------------------------------------------------------------- what surrounds a sub-layer
def read_streams(xs: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    """xs [S, T, D]; the sub-layer's input sum_s in[s] x_s."""
    return sum(w_in[s] * xs[s] for s in range(xs.shape[0]))


def write_streams(xs: torch.Tensor, mix: torch.Tensor, out: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """New streams from the old ones: x_t <- sum_s mix[s, t] x_s + out[t] y (mix is [from, to])."""
    S = xs.shape[0]
    return torch.stack([sum(mix[s, t] * xs[s] for s in range(S)) + out[t] * y for t in range(S)])


def token_shift(h: torch.Tensor, shift: torch.Tensor) -> torch.Tensor:
    """h_t + (h_(t-1) - h_t) * shift, with zeros before the first token and h_(t-1) as it was."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)
    return h + (before - h) * shift


def residual_gate(h: torch.Tensor, W: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    return torch.sigmoid(h @ W.T + b)


# ---------------------------------------------------------------- mixers
def query_temperature(T: int, coef: float, every: int, dtype) -> torch.Tensor:
    """One factor per position p: 1 + coef ln(floor((p + 1) / every) + 1)."""
    return torch.tensor([1.0 + coef * math.log((p + 1) // every + 1.0) for p in range(T)], dtype=dtype)


def causal_softmax_attention(q, k, v, scale: float, softcap: Optional[float]) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e]; query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    mask = torch.tril(torch.ones(T, T, dtype=torch.bool))
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(~mask, float("-inf"))
        out[:, h] = torch.softmax(s, dim=-1) @ v[:, h // rep]
    return out


def difference_factor(lq1, lk1, lq2, lk2, diff: float):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def differential_attention(x: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """Two attention maps per head over the same values; the second, times one learned number, is taken off the
    first, and the head's difference is divided by its root mean square and multiplied by 1 - diff."""
    T = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (x @ w[p + "q"].T + w[p + "q.b"]).view(T, H, 2, d)
    k = (x @ w[p + "k"].T + w[p + "k.b"]).view(T, G, 2, d)
    v = (x @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    if m.get("q_temp"):
        q = q * query_temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"], x.dtype).view(T, 1, 1, 1)
    a1 = causal_softmax_attention(q[:, :, 0], k[:, :, 0], v, m["scale"], m.get("softcap"))
    a2 = causal_softmax_attention(q[:, :, 1], k[:, :, 1], v, m["scale"], m.get("softcap"))
    lam = difference_factor(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    o = rms_unit(a1 - lam * a2, eps) * (1.0 - m["diff"])
    return o.reshape(T, H * dv) @ w[p + "o"].T + w[p + "o.b"]


def general_delta(x: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """Per head, with the unit key u: S <- diag(w) S - (a * u) (u^T S) + k v^T (both from the old S), o = S^T r."""
    T = x.shape[0]
    H, d = m["heads"], m["dim"]
    r, k, v = ((x @ w[p + n].T).view(T, H, d) for n in "rkv")
    z = torch.tanh(x @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(z)).view(T, H, d)
    a = torch.sigmoid(x @ w[p + "a"].T + w[p + "a.b"]).view(T, H, d)
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + UNIT_EPS)
    out = torch.zeros(T, H, d, dtype=x.dtype)
    S = torch.zeros(H, d, d, dtype=x.dtype)
    for t in range(T):
        read = torch.einsum("hk,hkv->hv", u[t], S)
        S = decay[t].unsqueeze(-1) * S - (a[t] * u[t]).unsqueeze(-1) * read.unsqueeze(1) + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out[t] = torch.einsum("hkv,hk->hv", S, r[t])
    o = rms_unit(out, eps).reshape(T, H * d) * w[p + "norm"] * torch.sigmoid(x @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward
def gated_dense(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def clamped_expert(h, gate, up, down, limit: float):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h: torch.Tensor, W: torch.Tensor, top: int, scale: float):
    """(chosen [T, top], their weights): softmax over all experts, the largest, times the scale as they are."""
    s = torch.softmax(h @ W.T, dim=-1)
    chosen = torch.topk(s, top, dim=-1).indices
    return chosen, torch.gather(s, 1, chosen) * scale


def router_margin(h: torch.Tensor, W: torch.Tensor, top: int) -> torch.Tensor:
    """Per token the gap between the last chosen expert's logit and the best one left out."""
    z = torch.sort(h @ W.T, dim=-1, descending=True).values
    return z[:, top - 1] - z[:, top] if top < z.shape[1] else torch.full((h.shape[0],), math.inf, dtype=h.dtype)


def mixture(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: dict, gaps_out: Optional[list] = None) -> torch.Tensor:
    r, limit = mlp["router"], mlp["expert"]["limit"]
    if gaps_out is not None:
        gaps_out.append(router_margin(h, w[p + "router"], r["top"]))
    chosen, weights = route(h, w[p + "router"], r["top"], r["scale"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        for t, j in (chosen == e).nonzero().tolist():
            out[t] += weights[t, j] * clamped_expert(h[t], w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"], limit)
    if mlp.get("shared"):
        s = clamped_expert(h, w[p + "shared.gate"], w[p + "shared.up"], w[p + "shared.down"], mlp["shared"]["limit"])
        out = out + s * torch.sigmoid(h @ w[p + "shared.sg"].T)
    return out


# ---------------------------------------------------------------- the model
def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            layers_out: Optional[list] = None, gaps_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence.  ``layers_out`` receives the sum of the streams after every
    layer, ``gaps_out`` every router's margin per token."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, T, D = cfg["norm"]["eps"], len(tokens), cfg["width"]
    x0 = w["embed"][torch.tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"] + sinusoids(T, D, dtype)
    xs = torch.stack([x0] * cfg["streams"])
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms_unit(read_streams(xs, w[p + "hc1.in"]), eps) * w[p + "norm1"]
        mixer = {"attention": differential_attention, "general_delta": general_delta}[layer["type"]]
        y = mixer(token_shift(h, w[p + "shift"]), w, p + "mix.", m, eps) * residual_gate(h, w[p + "rg1"], w[p + "rg1.b"])
        xs = write_streams(xs, w[p + "hc1.mix"], w[p + "hc1.out"], y)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms_unit(read_streams(xs, w[p + "hc2.in"]), eps) * w[p + "norm2"]
            y = gated_dense(h, w, p + "mlp.") if mlp["kind"] == "dense" else mixture(h, w, p + "mlp.", mlp, gaps_out)
            y = y * residual_gate(h, w[p + "rg2"], w[p + "rg2.b"])
            xs = write_streams(xs, w[p + "hc2.mix"], w[p + "hc2.out"], y)
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    x = rms_unit(xs.sum(0), eps) * w["final.norm"]
    return (x @ w["head"].T) * cfg["logit_scale"]


def decisive_tokens(cfg, w, tokens, seed, threshold=0.1, tries=2000):
    """``tokens`` with some of them drawn again until no router of the model meets a near-tie anywhere in the
    sequence (every margin above ``threshold``).  In 16-bit arithmetic a near-tie falls either way, and the row
    then differs by a whole expert; a comparison of logits wants prompts on which the design's answer does not
    hang on the last bit.  Tokens before the first near-tie stay as they are (the model is causal), so the search
    moves from left to right."""
    g = torch.Generator().manual_seed(seed)
    tokens = list(tokens)
    for _ in range(tries):
        gaps: list = []
        forward(cfg, w, tokens, gaps_out=gaps)
        if not gaps:
            return tokens
        close = (torch.stack(gaps).min(0).values < threshold).nonzero().flatten()
        if close.numel() == 0:
            return tokens
        tokens[int(close[0])] = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
    raise RuntimeError("no sequence without near-ties found")
