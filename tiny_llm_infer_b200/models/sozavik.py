"""Sozavik as data: which registered parts each layer is made of.

The stream starts as the embedding.  Every layer is a ``stream_*`` block: its sub-layers read the stream itself and only
their outputs are normed before the sum (an RMS norm with a plain gain).  The mixer is

* ``biased_attention`` with biases on q, k and v, normed queries and keys with gains shared by the heads, a rotation of
  neighbouring elements in part of every head (slow frequencies scaled down), a capped score, a sliding window, a learned
  sink and a gate of one number per head (layer type ``attention``);
* ``biased_attention`` with one norm over all heads of the queries and one over the keys, no positions and a sliding
  window (layer type ``attention_2``); or
* ``fixed_decay``, a linear recurrence with a constant decay per head over SiLU of q, k and v (layer type
  ``lightning``);

then, where the layer has one, a gated feed-forward with ReLU.  Among the attention layers that mix values the first
leaves its own to the later ones.  The head has its own matrix and a tanh cap on the logits.

Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.q|k|v`` (+ ``.b``) ``|q.norm|k.norm|vmix|sink|g|o``,
``l<i>.mix.q|k|v|g|o|norm``, ``l<i>.mlp.gate|up|down``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.sozavik import ARCHITECTURE, LightningConfig, RotatedAttentionConfig, SozavikConfig
from ..parts.spec import ExecEntry, LayerSpec, ModelDescription, PartSpec

FF_ACTIVATION = "relu"
GATED_NAMES = ("gate", "up", "down")
ATTENTION_NAMES = ("q", "k", "v", "o", "g")


def describe_sozavik(cfg: SozavikConfig) -> ModelDescription:
    layers = []

    def norm(prefix: str, name: str) -> PartSpec:
        return PartSpec("rmsnorm", dict(width=cfg.width, eps=cfg.norm_eps, name=name), prefix)

    mixed_before = False                          # whether a layer before has left its values
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if isinstance(m, LightningConfig):
            mixer = PartSpec("fixed_decay", dict(hidden_size=cfg.width, heads=m.heads, key_dim=m.dim, value_dim=m.vdim,
                                                 decays=m.decay, norm_eps=cfg.norm_eps), p + "mix.")
        else:
            common = dict(hidden_size=cfg.width, q_heads=m.heads, kv_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim,
                          scale=m.scale, window=m.window, unit_norm_eps=cfg.norm_eps, qk_gains=True, names=ATTENTION_NAMES)
            if m.v_mix:
                common["value_mix"] = "mix" if mixed_before else "first"
                mixed_before = True
            if isinstance(m, RotatedAttentionConfig):
                common.update(biases=True, output_bias=False, softcap=m.softcap, sink=True, learned_sink=True,
                              output_gate=True, gate_per_head=True)
                if m.rot_base is not None:
                    scaling = None if m.rot_scaling is None else m.rot_scaling.to_dict()
                    common["position"] = PartSpec("rotary_pairs", dict(head_dim=m.dim, theta=m.rot_base, rotary_dim=m.rot_dims,
                                                                       scaling=scaling))
            else:
                common["norm_whole"] = True
            mixer = PartSpec("biased_attention", common, p + "mix.")
        parts = {"mixer": mixer, "norm1": norm(p, "norm1")}
        block = "stream_mixer"
        if layer.mlp is not None:
            parts["ffn"] = PartSpec("swiglu", dict(hidden_size=cfg.width, intermediate_size=layer.mlp.ff,
                                                   activation=FF_ACTIVATION, names=GATED_NAMES), p + "mlp.")
            parts["norm2"] = norm(p, "norm2")
            block += "_ffn"
        layers.append(LayerSpec(block, parts))
    return ModelDescription(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=cfg.max_position_embeddings,
        embedding=PartSpec("token_embedding", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, name="embed"), ""),
        layers=tuple(layers),
        order=tuple(ExecEntry(i) for i in range(len(cfg.layers))),
        final_norm=norm("final.", "norm"),
        head=PartSpec("lm_head", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, tied=False, name="head",
                                      softcap=cfg.logit_softcap), ""),
    )


register_architecture(ARCHITECTURE, SozavikConfig, describe_sozavik, model_types=("sozavik",))
