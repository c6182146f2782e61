"""Several residual streams side by side ("hyper-connections") and what surrounds a sub-layer there.

The residual is x [T, S, D] float32, S streams.  A sub-layer q reads u = sum_s in[s] x_s through the model's norm,
h = norm(u), and its output y goes back to all streams at once, x_t <- sum_s mix[s, t] x_s + out[t] y; in, out and mix
are learned numbers of the sub-layer (``stream_mix``).  Two more parts stand between a norm and its sub-layer:

``residual_gate``   y is multiplied element by element by sigmoid(W h + b), h the norm's output (before any shift);
``token_shift``     the mixer reads h_t + (h_(t-1) - h_t) * shift, zeros before the first token; the previous token's h is
                    a state of the request (``StateSpec``), so this part is listed among its block's mixers and gets a
                    cache of its own.

The update of one sub-layer and the read of the next are one kernel (``ops.stream_read``): a block hands its last output
on as a ``StreamUpdate``, and the norm that follows (``stream_norm``) updates, reads, norms and shifts.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import torch

from .. import ops
from .registry import register
from .spec import CacheSpec, ParamSpec, StateSpec


@dataclass
class StreamUpdate:
    """The streams x [T, S * D] and a sub-layer's output that is still to be mixed into them (none: ``delta`` None)."""
    x: torch.Tensor
    delta: Optional[torch.Tensor] = None
    delta_bias: Optional[torch.Tensor] = None      # float32 [D]: a bias of the sub-layer's last product
    gate: Optional[torch.Tensor] = None            # logits [T, D]
    gate_bias: Optional[torch.Tensor] = None       # float32 [D]
    mix: Optional["StreamMix"] = None


@register("norm", "stream_mix")
class StreamMix:
    """A sub-layer's weights on the streams: ``in`` [S] (read), ``out`` [S] (write) and ``mix`` [S, S] (from, to).  It has
    no ``forward``: the norm that follows the sub-layer applies it."""

    def __init__(self, streams: int, dtype: torch.dtype, device, names=("in", "out", "mix")):
        self.streams, self.dtype, self.device, self.names = int(streams), dtype, device, tuple(names)
        self.w_in = self.w_out = self.w_mix = None

    @classmethod
    def param_specs(cls, streams: int, names=("in", "out", "mix")) -> Dict[str, ParamSpec]:
        n_in, n_out, n_mix = names
        return {n_in: ParamSpec((streams,), "unit"), n_out: ParamSpec((streams,), "unit"),
                n_mix: ParamSpec((streams, streams), "unit")}

    def load(self, t: Dict[str, torch.Tensor]) -> None:
        self.w_in, self.w_out, self.w_mix = (t[n].to(torch.float32).contiguous() for n in self.names)


@register("norm", "residual_gate")
class ResidualGate:
    """Logits of the gate on a sub-layer's output, W h in the storage type; the bias and the sigmoid are applied where
    the output meets the streams."""

    def __init__(self, width: int, dtype: torch.dtype, device, name: str = "weight", bias_suffix: str = ".b"):
        self.width, self.dtype, self.device, self.name, self.bias_suffix = int(width), dtype, device, name, bias_suffix
        self.weight = self.bias = None

    @classmethod
    def param_specs(cls, width: int, name: str = "weight", bias_suffix: str = ".b") -> Dict[str, ParamSpec]:
        return {name: ParamSpec((width, width)), name + bias_suffix: ParamSpec((width,), "unit")}

    def load(self, t: Dict[str, torch.Tensor]) -> None:
        self.weight = t[self.name].contiguous()
        self.bias = t[self.name + self.bias_suffix].to(torch.float32).contiguous()

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return ops.linear(h, self.weight, out_dtype=self.dtype)


@register("mixer", "token_shift")
class TokenShift:
    """The learned weights of a shift by one token and its state, the previous token's h.  The norm's kernel applies it."""
    graph_safe = True

    def __init__(self, width: int, dtype: torch.dtype, device, name: str = "shift"):
        self.width, self.dtype, self.device, self.name = int(width), dtype, device, name
        self.weight: Optional[torch.Tensor] = None

    @classmethod
    def param_specs(cls, width: int, name: str = "shift") -> Dict[str, ParamSpec]:
        return {name: ParamSpec((int(width),), "norm")}

    def load(self, t: Dict[str, torch.Tensor]) -> None:
        self.weight = t[self.name].to(torch.float32).contiguous()

    def cache_spec(self) -> Optional[CacheSpec]:
        return None

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((self.width,), "float32")


@register("norm", "stream_norm")
class StreamNorm:
    """RMS norm of a weighted sum of the streams, with the update that precedes it.  ``gain_scale``: a constant that the
    gain is multiplied by (a factor of whatever reads the norm's output linearly, such as the logits)."""

    def __init__(self, width: int, streams: int, eps: float, dtype: torch.dtype, device, name: str = "weight",
                 gain_scale: float = 1.0):
        self.width, self.streams, self.eps, self.dtype, self.device = int(width), int(streams), float(eps), dtype, device
        self.name, self.gain_scale = name, float(gain_scale)
        self.gain: Optional[torch.Tensor] = None

    @classmethod
    def param_specs(cls, width: int, streams: int, eps: float, name: str = "weight", gain_scale: float = 1.0) -> Dict[str, ParamSpec]:
        return {name: ParamSpec((int(width),), "norm")}

    def load(self, t: Dict[str, torch.Tensor]) -> None:
        self.gain = (t[self.name].to(torch.float32) * self.gain_scale).contiguous()

    def workspace_floats(self, tokens: int) -> int:
        return 2 * tokens * self.streams * self.width          # the streams before and after an update

    def _read(self, update: StreamUpdate, **more):
        u = update
        mix = u.mix
        return ops.stream_read(u.x, self.streams, self.gain, self.eps, self.dtype, delta=u.delta, delta_bias=u.delta_bias,
                               gate=u.gate, gate_bias=u.gate_bias, mix=None if mix is None else mix.w_mix,
                               w_out=None if mix is None else mix.w_out, **more)

    def read(self, update: StreamUpdate, mix: StreamMix, ctx=None, shift: Optional[TokenShift] = None, tail=None):
        """(streams after the update, h, what the sub-layer reads): h itself, or, with ``shift``, h shifted by a token."""
        if shift is None:
            x, h, _ = self._read(update, w_in=mix.w_in)
            return x, h, h
        return self._read(update, w_in=mix.w_in, shift=shift.weight, tail=tail, token_slot=ctx.token_slot,
                          seg_info=ctx.seg_info, single_tokens=ctx.decode_only)

    def forward(self, h: torch.Tensor, delta, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """The model's last norm: of the plain sum of the streams."""
        update = delta if isinstance(delta, StreamUpdate) else StreamUpdate(h)
        return self._read(update, rows=rows)[1]
