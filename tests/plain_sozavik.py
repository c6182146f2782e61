"""Sozavik, plainly: whole sequences, no cache, no batching, float64 unless told otherwise; one
function per mechanism.  It shares no code with the engine and is what the engine is compared with.

``weights`` maps tensor names to torch tensors (any float type), ``cfg`` is the dictionary of
config.json.  Notation: T tokens, D the model width, rows are tokens.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------- positions
def frequencies(dims: int, base: float, scaling: Optional[dict]) -> List[float]:
    """One frequency per rotated pair.  With ``scaling`` the slow ones (few turns within the original length) are
    divided by the factor, the fast ones stay, and those between are blended by where their turns fall."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wave = 2.0 * math.pi / f
            orig, low, high, factor = (float(scaling[k]) for k in ("original", "low", "high", "factor"))
            if wave > orig / low:
                f = f / factor
            elif not wave < orig / high:
                s = (orig / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate_pairs(x: torch.Tensor, freqs: List[float], first: int = 0) -> torch.Tensor:
    """x [T, heads, d], row t at position ``first`` + t: elements 2i and 2i + 1 turn together by position * freqs[i]."""
    out = x.clone()
    p = torch.arange(first, first + x.shape[0], dtype=torch.float64)
    for i, f in enumerate(freqs):
        c, s = (fn(p * f).to(x.dtype).view(-1, 1) for fn in (torch.cos, torch.sin))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ---------------------------------------------------------------- attention
def softmax_attention(q, k, v, scale: float, softcap: Optional[float], window: Optional[int],
                      sink: Optional[torch.Tensor]) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e]; query head h reads key/value head h // (H / G).  Row i sees the rows
    j with 0 <= i - j < window; ``sink`` [H] is one more score per head, of a key that carries nothing."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    back = torch.arange(T).view(T, 1) - torch.arange(T).view(1, T)
    seen = (back >= 0) & (back < (window or T + 1))
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(~seen, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink[h].expand(T, 1)], dim=1)
        out[:, h] = torch.softmax(s, dim=-1)[:, :T] @ v[:, h // rep]
    return out


def mixed_values(v: torch.Tensor, first: Optional[torch.Tensor], share: torch.Tensor) -> torch.Tensor:
    """(1 - share) v + share first; the first layer that mixes has nothing to mix with."""
    return v if first is None else (1.0 - share) * v + share * first


def rotated_attention(x, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, first_values=None):
    """Type ``attention``; returns (output, values before any mixing)."""
    T, H, G, d, e = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (x @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d)
    k = (x @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d)
    v = (x @ w[p + "v"].T + w[p + "v.b"]).view(T, G, e)
    q = rms_unit(q, eps) * w[p + "q.norm"]
    k = rms_unit(k, eps) * w[p + "k.norm"]
    if m.get("rot"):
        f = frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        q, k = rotate_pairs(q, f), rotate_pairs(k, f)
    mixed = mixed_values(v, first_values, w[p + "vmix"]) if m.get("v_mix") else v
    o = softmax_attention(q, k, mixed, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"), w[p + "sink"])
    o = o * torch.sigmoid(x @ w[p + "g"].T).unsqueeze(-1)
    return o.reshape(T, H * e) @ w[p + "o"].T, v


def whole_normed_attention(x, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, first_values=None):
    """Type ``attention_2``; returns (output, values before any mixing)."""
    T, H, G, d, e = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms_unit(x @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, d)
    k = (rms_unit(x @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, d)
    v = (x @ w[p + "v"].T).view(T, G, e)
    mixed = mixed_values(v, first_values, w[p + "vmix"]) if m.get("v_mix") else v
    o = softmax_attention(q, k, mixed, m["scale"], None, (m.get("mask") or {}).get("size"), None)
    return o.reshape(T, H * e) @ w[p + "o"].T, v


# ---------------------------------------------------------------- recurrence
def fixed_decay_recurrence(q, k, v, decay) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, e], one decay per head: S <- decay S + k v^T, o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    a = torch.tensor(decay, dtype=q.dtype).view(H, 1, 1)
    for t in range(T):
        S = a * S + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out


def lightning(x, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H = x.shape[0], m["heads"]
    q, k, v = (silu(x @ w[p + n].T).view(T, H, -1) for n in "qkv")
    o = fixed_decay_recurrence(q, k, v, m["decay"]).reshape(T, -1)
    o = rms_unit(o, eps) * w[p + "norm"] * torch.sigmoid(x @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward
def relu_unit(x, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (torch.relu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


# ---------------------------------------------------------------- the model
def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence.  ``layers_out`` receives the stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    first = None                                  # values of the first layer that mixes
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "lightning":
            y = lightning(x, w, p + "mix.", m, eps)
        else:
            attend = {"attention": rotated_attention, "attention_2": whole_normed_attention}[layer["type"]]
            y, v = attend(x, w, p + "mix.", m, eps, first)
            if first is None and m.get("v_mix"):
                first = v
        x = x + rms_unit(y, eps) * w[p + "norm1"]
        if layer.get("mlp") is not None:
            x = x + rms_unit(relu_unit(x, w, p + "mlp."), eps) * w[p + "norm2"]
        if layers_out is not None:
            layers_out.append(x)
    logits = (rms_unit(x, eps) * w["final.norm"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits
