"""Vigonex as data: which registered parts each layer is made of.

The stream starts as the scaled embedding plus the position's sinusoids, once per residual stream.  Every layer is a
``hyper_*_gated_shifted`` block: each sub-layer reads a learned weighted sum of the streams through an RMS norm and is
written back to all of them with a learned mix, its output multiplied by a residual gate; the mixer's input is shifted by
a token.  The mixer is

* ``biased_attention`` with two maps per head over the same values (``differential``), biases, a query temperature and a
  capped score (layer type ``attention``), or
* ``erase_delta``, the delta rule with a decay and a removal rate per head and key channel (layer type
  ``general_delta``);

then, where the layer has one, a ``swiglu`` feed-forward with SiLU, or a mixture of clamped-swish experts weighted by the
softmax over all of them, with a shared expert under a gate of one number per token.  The model's last norm reads the
plain sum of the streams; its gain carries the logits' scale.

Tensor names: ``embed``, ``l<i>.norm1|norm2|shift|rg1|rg1.b|rg2|rg2.b``, ``l<i>.hc1|hc2.in|out|mix``,
``l<i>.mix.q|k|v|o`` (+ ``.b``) ``|lq1|lk1|lq2|lk2``, ``l<i>.mix.r|k|v|g|a|a.b|w1|w2|w0|norm|o``, ``l<i>.mlp.gate|up|down``,
``l<i>.mlp.router``, ``l<i>.mlp.e<j>.gate|up|down``, ``l<i>.mlp.shared.gate|up|down|sg``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import math

from ..config.base import register_architecture
from ..config.vigonex import ARCHITECTURE, DenseConfig, DifferentialConfig, VigonexConfig, default_rank
from ..parts.spec import ExecEntry, LayerSpec, ModelDescription, PartSpec

POSITION_BASE = 10000.0       # of the sinusoids' frequencies
UNIT_EPS = 1e-6               # under the root when the delta rule's key is made a unit vector
DECAY_RATE = math.exp(-0.5)   # the delta rule's decay is exp(-DECAY_RATE sigmoid(.))
SWISH_SLOPE = 1.702           # of the experts' gate, g sigmoid(slope g)
GATED_NAMES = ("gate", "up", "down")
ATTENTION_NAMES = ("q", "k", "v", "o", "g")


def describe_vigonex(cfg: VigonexConfig) -> ModelDescription:
    layers = []

    def norm(prefix: str, name: str, **more) -> PartSpec:
        return PartSpec("stream_norm", dict(width=cfg.width, streams=cfg.streams, eps=cfg.norm_eps, name=name, **more), prefix)

    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        if isinstance(m, DifferentialConfig):
            mixer = PartSpec("biased_attention", dict(
                hidden_size=cfg.width, q_heads=m.heads, kv_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim, scale=m.scale,
                softcap=m.softcap, q_temperature=None if m.temp_every is None else (m.temp_coef, m.temp_every), biases=True,
                defer_output_bias=True, differential=(m.diff, cfg.norm_eps), names=ATTENTION_NAMES), p + "mix.")
        else:
            mixer = PartSpec("erase_delta", dict(
                hidden_size=cfg.width, heads=m.heads, key_dim=m.dim, value_dim=m.dim,
                decay_rank=m.decay_rank or default_rank(cfg.width), norm_eps=cfg.norm_eps, decay_rate=DECAY_RATE,
                unit_eps=UNIT_EPS), p + "mix.")
        parts = {"norm1": norm(p, "norm1"), "hc1": PartSpec("stream_mix", dict(streams=cfg.streams), p + "hc1."),
                 "shift": PartSpec("token_shift", dict(width=cfg.width, name="shift"), p),
                 "gate1": PartSpec("residual_gate", dict(width=cfg.width, name="rg1"), p), "mixer": mixer}
        block = "hyper_mixer"
        if layer.mlp is not None:
            block += "_ffn"
            f = layer.mlp
            parts["norm2"] = norm(p, "norm2")
            parts["hc2"] = PartSpec("stream_mix", dict(streams=cfg.streams), p + "hc2.")
            parts["gate2"] = PartSpec("residual_gate", dict(width=cfg.width, name="rg2"), p)
            if isinstance(f, DenseConfig):
                parts["ffn"] = PartSpec("swiglu", dict(hidden_size=cfg.width, intermediate_size=f.ff, activation="silu",
                                                       names=GATED_NAMES), p + "mlp.")
            else:
                shared = None
                if f.shared_ff is not None:
                    shared = PartSpec("swiglu", dict(hidden_size=cfg.width, intermediate_size=f.shared_ff,
                                                     activation="clamped_swish", act_consts=(f.shared_limit, SWISH_SLOPE),
                                                     names=GATED_NAMES), "shared.")
                parts["ffn"] = PartSpec("moe", dict(
                    hidden_size=cfg.width, experts=f.experts, top=f.top, expert_size=f.expert_ff, activation="clamped_swish",
                    act_consts=(f.expert_limit, SWISH_SLOPE), router_scores="softmax_all", router_scale=f.router_scale,
                    weight_on="output", names=GATED_NAMES, shared=shared,
                    shared_gate=None if shared is None else "sg"), p + "mlp.")
        layers.append(LayerSpec(block + "_gated_shifted", parts))
    return ModelDescription(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=cfg.max_position_embeddings,
        embedding=PartSpec("sinusoid_embedding", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, scale=cfg.embedding_scale,
                                                      name="embed", base=POSITION_BASE, streams=cfg.streams), ""),
        layers=tuple(layers),
        order=tuple(ExecEntry(i) for i in range(len(cfg.layers))),
        final_norm=norm("final.", "norm", gain_scale=cfg.logit_scale),
        head=PartSpec("lm_head", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, tied=False, name="head"), ""),
    )


register_architecture(ARCHITECTURE, VigonexConfig, describe_vigonex, model_types=("vigonex",))
