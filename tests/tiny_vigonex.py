"""Tiny Vigonex configurations for the tests.  They differ in every size and constant and take values that hide nothing:
one to five residual streams, layers in every order (attention first, the delta rule first, either alone), layers
without a feed-forward, dense ones and mixtures with and without a shared expert, fewer key/value heads than query heads
and one head alone, value widths below, equal to and above a map's key width, with and without a temperature and a cap,
ranks and widths on and off the vector kernels' multiples of eight, an odd width (the last sinusoid has no cosine),
scales of one and others, limits of the shared expert and of the routed ones that differ.

The weights are then shaped so that every mechanism shows: mixes of the streams near a permutation plus noise, gates
and shifts spread out, routers decisive, gate and up sums wide enough that the limits bite, the difference's learned
number well away from its constant, and half of the delta rule's heads slow to forget and to be overwritten, so that
what was written hundreds of tokens ago still shows in the read-out."""
from __future__ import annotations

import tempfile
from dataclasses import replace
from pathlib import Path

import torch

from tiny_llm_infer_b200.config.vigonex import (DenseConfig, DifferentialConfig, GeneralDeltaConfig, MixtureConfig,
                                                VigonexConfig, VigonexLayerConfig)
from tiny_llm_infer_b200.weights import write_random_model
from tiny_llm_infer_b200.weights.safetensors_io import SafetensorsFile, save_file


def att(heads, kv_heads, dim, vdim, scale, diff, cap, temp=None, mlp=None):
    coef, every = temp or (0.0, None)
    return VigonexLayerConfig("attention", DifferentialConfig(heads, kv_heads, dim, vdim, scale, diff, cap, coef, every), mlp)


def delta(heads, dim, rank, mlp=None):
    return VigonexLayerConfig("general_delta", GeneralDeltaConfig(heads, dim, rank), mlp)


def moe(ff, limit, experts, top, scale, shared=None):
    return MixtureConfig(ff, limit, experts, top, scale, *(shared or (None, None)))


# multiples of eight: the vector kernels and, in bfloat16, the tensor-core attention; three streams
G1 = dict(cfg=VigonexConfig(vocab=320, width=128, streams=3, norm_eps=1e-5, embedding_scale=2.0, logit_scale=0.5, layers=(
    att(6, 2, 24, 40, 0.3, 0.3, 9.0, (0.4, 16), mlp=moe(48, 0.8, 6, 2, 1.5, (64, 1.2))),
    delta(4, 16, 8, mlp=DenseConfig(96)),
    att(3, 3, 16, 16, 0.4, 0.7, None, (0.2, 50)),
    delta(2, 40, 16, mlp=moe(40, 1.5, 5, 3, 1.0)),
)), seed=61, std=0.1, norm_range=(0.7, 1.3), page_size=16, lengths=(70, 97, 130, 41, 66, 35))
# nothing a multiple of eight, an odd width, one stream, one head alone, pages of 8
G2 = dict(cfg=VigonexConfig(vocab=401, width=101, streams=1, norm_eps=3e-6, embedding_scale=1.0, logit_scale=1.0, layers=(
    delta(3, 10, 5, mlp=moe(30, 1.1, 4, 1, 2.5, (22, 0.6))),
    att(1, 1, 10, 6, 0.5, 0.2, 4.0, (0.8, 7), mlp=DenseConfig(50)),
    delta(1, 22, 3),
    att(4, 1, 6, 22, 0.6, 0.45, None, mlp=moe(18, 0.7, 7, 4, 0.8)),
)), seed=62, std=0.14, norm_range=(0.6, 1.4), page_size=8, lengths=(70, 97, 41, 35, 66))
# the tensor-core kernels' own widths (maps of 64 with values of 128, maps of 128 with values of 64), states of 128 rows,
# pages of 32, prompts of hundreds of tokens; four streams
G3 = dict(cfg=VigonexConfig(vocab=512, width=192, streams=4, norm_eps=1e-6, embedding_scale=0.5, logit_scale=2.0, layers=(
    att(4, 2, 64, 128, 0.12, 0.8, 20.0, (0.35, 64), mlp=moe(64, 2.0, 8, 2, 1.2, (80, 0.9))),
    delta(2, 128, 24, mlp=moe(56, 1.0, 12, 3, 2.0, (40, 1.4))),
    att(8, 1, 128, 64, 0.08, 0.35, 40.0, (0.5, 100), mlp=DenseConfig(136)),
)), seed=63, std=0.08, norm_range=(0.8, 1.2), page_size=32, lengths=(70, 230, 130, 41, 150, 35))
# the delta rule alone (no pages at all), five streams (the kernel for any number of them), a width of its own
G4 = dict(cfg=VigonexConfig(vocab=300, width=88, streams=5, norm_eps=1e-5, embedding_scale=3.5, logit_scale=0.3, layers=(
    delta(2, 24, 7, mlp=DenseConfig(40)),
    delta(5, 12, 8),
)), seed=64, std=0.12, norm_range=(0.7, 1.3), page_size=16, lengths=(70, 97, 41, 35, 66))
VIGONEXES = {"G1": G1, "G2": G2, "G3": G3, "G4": G4}


def slow_heads(w0: torch.Tensor, a_bias: torch.Tensor, heads: int):
    """Every second head's decay near exp(-0.001) and its removal rate near a hundredth per token."""
    w0, a_bias = w0.clone().view(heads, -1), a_bias.clone().view(heads, -1)
    w0[::2] -= 6.5
    a_bias[::2] -= 4.5
    return w0.reshape(-1), a_bias.reshape(-1)


def make_folder(tiny, folder=None, dtype=torch.bfloat16) -> Path:
    folder = Path(folder or tempfile.mkdtemp(prefix="tllm_vigo_"))
    write_random_model(folder, tiny["cfg"], tiny["seed"], tiny["std"], tiny["norm_range"], dtype=dtype)
    f = SafetensorsFile(folder / "model.safetensors")
    tensors = {name: f.read(name).clone() for name in f.tensors}
    f.close()
    cfg, g = tiny["cfg"], torch.Generator().manual_seed(tiny["seed"])
    S, unit = cfg.streams, 1.0 / tiny["std"] / cfg.width ** 0.5        # times this, a product's outputs have order one

    def change(name, fn):
        tensors[name] = fn(tensors[name].float()).to(dtype)

    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        for q in ("1", "2") if layer.mlp is not None else ("1",):
            turned = torch.eye(S).roll(1, 0) * 0.5 + torch.eye(S) * 0.5 if q == "1" else torch.eye(S)
            change(p + f"hc{q}.mix", lambda m: turned + 0.15 * torch.randn(S, S, generator=g))
            change(p + f"hc{q}.in", lambda v: 0.7 + 0.5 * torch.rand(S, generator=g) * (-1.0) ** torch.arange(S))
            change(p + f"hc{q}.out", lambda v: 0.6 + 0.8 * torch.rand(S, generator=g))
            change(p + f"rg{q}", lambda v: v * unit * 1.5)
        change(p + "shift", lambda v: torch.rand(cfg.width, generator=g) * 1.2 - 0.2)
        if layer.type == "attention":
            for n in ("lq1", "lk1", "lq2", "lk2"):
                change(p + "mix." + n, lambda v: torch.randn(v.shape, generator=g) * 0.3)
            change(p + "mix.q", lambda v: v * unit * 1.5)
            change(p + "mix.k", lambda v: v * unit * 1.5)
        else:
            a, b = slow_heads(tensors[p + "mix.w0"].float(), tensors[p + "mix.a.b"].float(), layer.mixer.heads)
            tensors[p + "mix.w0"], tensors[p + "mix.a.b"] = a.to(dtype), b.to(dtype)
            for n in ("r", "k", "v", "g", "a", "w1"):
                change(p + "mix." + n, lambda v: v * unit)
            change(p + "mix.w2", lambda v: v / tiny["std"] / v.shape[1] ** 0.5 * 0.7)
        if isinstance(layer.mlp, MixtureConfig):
            change(p + "mlp.router", lambda r: r * unit * 5.0)          # logits of order five
            for n in list(tensors):
                if n.startswith(p + "mlp.") and n.rsplit(".", 1)[1] in ("gate", "up", "sg"):
                    change(n, lambda v: v * unit * 1.3)
    save_file(tensors, folder / "model.safetensors")
    return folder


def as_read(cfg: VigonexConfig) -> VigonexConfig:
    """``cfg`` without what config.json does not carry (the ranks)."""
    return replace(cfg, layers=tuple(replace(l, mixer=replace(l.mixer, decay_rank=None)) if l.type == "general_delta" else l
                                     for l in cfg.layers))


def prompt(seed: int, length: int, vocab: int):
    g = torch.Generator().manual_seed(9000 + seed)
    return torch.randint(0, vocab, (length,), generator=g).tolist()


def requests_for(tiny):
    return {str(i): prompt(i, n, tiny["cfg"].vocab) for i, n in enumerate(tiny["lengths"])}
