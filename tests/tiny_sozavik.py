"""Tiny Sozavik configurations for the tests.  They differ in every size and constant and take values that hide nothing:
layers in every order (either attention or the recurrence first), with and without a feed-forward, windows shorter than a
page, no multiple of one and none at all, fewer key/value heads than query heads and one head alone, value widths below,
equal to and above the keys', rotations of part of a head and of all of it, with scaled slow frequencies, without and no
rotation at all, scores with and without a cap, logits with and without one; the first layer that mixes values of either
type, with layers that do not mix before, between and after; key widths of the recurrence above and below its value
widths, and widths on and off the vector and tensor-core kernels.

The weights are then shaped so that every mechanism shows: scores of several units, sinks that hold a good share of the
weight, mixing shares and gates spread out, and heads of the recurrence from a few tokens to hundreds."""
from __future__ import annotations

import tempfile
from pathlib import Path

import torch

from tiny_llm_infer_b200.config.sozavik import (DenseConfig, FrequencyScaling, LightningConfig, RotatedAttentionConfig,
                                                SozavikConfig, SozavikLayerConfig, WholeNormAttentionConfig)
from tiny_llm_infer_b200.weights import write_random_model
from tiny_llm_infer_b200.weights.safetensors_io import SafetensorsFile, save_file


def rotated(heads, kv, dim, vdim, scale, cap, window, rot=None, scaling=None, v_mix=False, ff=None):
    base, dims = rot or (None, 0)
    return SozavikLayerConfig("attention", RotatedAttentionConfig(
        heads, kv, dim, vdim, scale, cap, window, base, dims, None if scaling is None else FrequencyScaling(*scaling), v_mix),
        None if ff is None else DenseConfig(ff))


def whole(heads, kv, dim, vdim, scale, window, v_mix=False, ff=None):
    return SozavikLayerConfig("attention_2", WholeNormAttentionConfig(heads, kv, dim, vdim, scale, window, v_mix),
                              None if ff is None else DenseConfig(ff))


def lightning(dim, vdim, decay, ff=None):
    return SozavikLayerConfig("lightning", LightningConfig(len(decay), dim, vdim, tuple(decay)),
                              None if ff is None else DenseConfig(ff))


# multiples of eight: the vector kernels and, in bfloat16, the tensor-core attention; the whole-normed layer mixes first
Z1 = dict(cfg=SozavikConfig(vocab=320, width=128, norm_eps=1e-5, logit_softcap=8.0, layers=(
    whole(4, 4, 32, 16, 0.35, 40, ff=160),
    whole(6, 2, 24, 40, 0.3, 25, v_mix=True, ff=96),
    lightning(16, 24, (0.999, 0.7, 0.95)),
    rotated(4, 2, 40, 40, 0.25, 9.0, 21, rot=(500.0, 24), scaling=(4.0, 1.0, 4.0, 64.0), v_mix=True, ff=64),
    rotated(8, 2, 16, 40, 0.5, None, None, rot=(10000.0, 16), v_mix=True),
)), seed=71, std=0.1, norm_range=(0.7, 1.3), page_size=16, lengths=(70, 97, 130, 41, 66, 35))
# nothing a multiple of eight, one head alone, pages of 8, windows shorter than a page; the rotated layer mixes first
Z2 = dict(cfg=SozavikConfig(vocab=401, width=101, norm_eps=3e-6, logit_softcap=None, layers=(
    lightning(10, 6, (0.9, 0.99, 0.4, 1.0), ff=50),
    rotated(3, 1, 10, 6, 0.9, 4.0, 5, rot=(77.0, 4), scaling=(8.0, 1.5, 3.0, 40.0), v_mix=True, ff=30),
    whole(1, 1, 22, 6, 0.4, 13, v_mix=True),
    rotated(5, 5, 12, 20, 0.5, None, 33, v_mix=False, ff=46),
    whole(7, 1, 6, 6, 0.8, None, v_mix=True, ff=22),
)), seed=72, std=0.13, norm_range=(0.6, 1.4), page_size=8, lengths=(70, 97, 41, 35, 66))
# the tensor-core kernels' own widths (keys and values of 128 without a cap or a gate take the tcgen05 prompt kernel),
# pages of 32, prompts of hundreds of tokens
Z3 = dict(cfg=SozavikConfig(vocab=512, width=192, norm_eps=1e-6, logit_softcap=20.0, layers=(
    rotated(4, 2, 64, 128, 0.12, 30.0, 150, rot=(20.0, 32), scaling=(2.0, 2.0, 6.0, 300.0), v_mix=True, ff=256),
    whole(4, 2, 128, 128, 0.1, 100, v_mix=True, ff=136),
    lightning(128, 64, (0.98, 0.998), ff=96),
    whole(2, 1, 128, 128, 0.15, 64, ff=64),
    rotated(8, 2, 128, 128, 0.09, 50.0, 70, rot=(1e6, 128), v_mix=True),
)), seed=73, std=0.08, norm_range=(0.8, 1.2), page_size=32, lengths=(70, 300, 130, 41, 210, 35))
# the recurrence alone (no pages at all)
Z4 = dict(cfg=SozavikConfig(vocab=300, width=88, norm_eps=1e-5, logit_softcap=5.0, layers=(
    lightning(24, 40, (0.97, 0.8), ff=40),
    lightning(12, 8, (0.6, 0.9, 0.99, 0.999, 1.0)),
)), seed=74, std=0.12, norm_range=(0.7, 1.3), page_size=16, lengths=(70, 97, 41, 35, 66))
SOZAVIKS = {"Z1": Z1, "Z2": Z2, "Z3": Z3, "Z4": Z4}


def make_folder(tiny, folder=None, dtype=torch.bfloat16) -> Path:
    folder = Path(folder or tempfile.mkdtemp(prefix="tllm_soza_"))
    write_random_model(folder, tiny["cfg"], tiny["seed"], tiny["std"], tiny["norm_range"], dtype=dtype)
    f = SafetensorsFile(folder / "model.safetensors")
    tensors = {name: f.read(name).clone() for name in f.tensors}
    f.close()
    cfg, g = tiny["cfg"], torch.Generator().manual_seed(tiny["seed"])
    unit = 1.0 / tiny["std"] / cfg.width ** 0.5              # times this, a product's outputs have the input's spread

    def change(name, fn):
        tensors[name] = fn(tensors[name].float()).to(dtype)

    change("embed", lambda v: v / tiny["std"])
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}.mix."
        for n in "qkvg":
            if p + n in tensors:
                change(p + n, lambda v: v * unit)
        if p + "vmix" in tensors:
            change(p + "vmix", lambda v: 0.3 + 0.4 * torch.rand((), generator=g))
        if p + "sink" in tensors:
            change(p + "sink", lambda v: 1.0 + 1.5 * torch.randn(v.shape, generator=g))
        for n in ("q.norm", "k.norm"):                       # scores of a few units
            if p + n in tensors:
                change(p + n, lambda v: v * (2.0 / layer.mixer.scale / layer.mixer.dim ** 0.5) ** 0.5)
        if layer.mlp is not None:
            for n in ("gate", "up"):
                change(f"l{i}.mlp.{n}", lambda v: v * unit)
    save_file(tensors, folder / "model.safetensors")
    return folder


def prompt(seed: int, length: int, vocab: int):
    g = torch.Generator().manual_seed(12000 + seed)
    return torch.randint(0, vocab, (length,), generator=g).tolist()


def requests_for(tiny):
    return {str(i): prompt(i, n, tiny["cfg"].vocab) for i, n in enumerate(tiny["lengths"])}
