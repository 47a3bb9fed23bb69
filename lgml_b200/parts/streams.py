"""A residual in several streams ("hyper-connections") and a gate on what every sublayer adds.

Instead of one residual x there are R streams x_1 .. x_R, all equal to the embedding's rows at the start.  For
every sublayer, with its own weights in [R], out [R] and mix [R, R]:

    h    = norm(sum_s in[s] x_s)
    y    = sublayer(h) [* sigmoid(W_g h + b_g)]
    x_t  = sum_s mix[s, t] x_s + out[t] y            all streams at once from the old ones

and after the last layer x is the sum of the streams.  What a sublayer computed, its gate and the update of the
streams are not applied on their own: the block hands them on as a ``PendingStreams``, and the next norm (the next
sublayer's, or the model's final one) does the gate, the update, the sum it reads and its norm in one kernel.

The gate's projection reads what the sublayer reads, so its rows are stacked in front of the sublayer's own
in-projection when the sublayer can be given one (``in_rows`` / ``forward_projected``): one product for both.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..weights import VECTOR, TensorSpec
from .base import Part, register_part
from .norm import RMSNorm


@dataclass
class PendingStreams:
    """What is still to happen to the streams: they start from ``start`` (times ``start_scale``), or a sublayer's result
    ``delta`` (float32 tensor or ``ops.Partials``) passes its gate (the logits; None: none) and updates them."""

    start: Optional[torch.Tensor] = None
    start_scale: float = 1.0
    delta: object = None
    gate: Optional[torch.Tensor] = None
    w_out: Optional[torch.Tensor] = None
    mix: Optional[torch.Tensor] = None


class StreamNorm(RMSNorm):
    """RMS norm of a weighted sum of the streams x [tokens, R, E], after what is pending for them."""

    takes_streams = True

    def forward(self, rt, x, out_dtype, delta=None, rows=None, w_in=None):
        """``delta``: a ``PendingStreams`` or None; ``w_in`` float32 [R] (None: the plain sum)."""
        n = x.shape[0] if rows is None else rows.numel()
        out = torch.empty((n, self.width), dtype=out_dtype, device=x.device)
        p = delta if delta is not None else PendingStreams()
        return ops.stream_norm(x, self.eps, out, self.weight, w_in=w_in, start=p.start, start_scale=p.start_scale, delta=p.delta, gate=p.gate,
                               w_out=p.w_out, mix=p.mix, rows=rows)


class Hyper(Part):
    """The three weights of one sublayer's connection to the streams: ``.in`` [R], ``.out`` [R], ``.mix`` [R, R] (from, to)."""

    graph_safe = True

    def __init__(self, streams: int):
        self.streams = streams
        self.w_in = self.w_out = self.mix = None

    def tensor_specs(self, prefix):
        R = self.streams
        return [TensorSpec(prefix + ".in", (R,), VECTOR, init=(1.0, 1.0)), TensorSpec(prefix + ".out", (R,), VECTOR, init=(1.0, 1.0)),
                TensorSpec(prefix + ".mix", (R, R), VECTOR, init=(1.0 / R, 1.0))]

    def bind(self, prefix, tensors, rt):
        self.w_in, self.w_out, self.mix = (tensors[prefix + n].float().contiguous() for n in (".in", ".out", ".mix"))


class ResultGate(Part):
    """sigmoid(W h + b) on a sublayer's result, h being what the sublayer reads.  Tensors: the prefix itself and ``.b``."""

    graph_safe = True

    def __init__(self, width: int):
        self.width = width
        self.w = self.b = None

    def tensor_specs(self, prefix):
        return [TensorSpec(prefix, (self.width, self.width)), TensorSpec(prefix + ".b", (self.width,), VECTOR)]

    def bind(self, prefix, tensors, rt):
        self.w, self.b = tensors[prefix], tensors[prefix + ".b"].float().contiguous()


class HyperBlock(Part):
    """A pre-norm layer on several streams: mixer, then (unless None) feed-forward, each optionally gated."""

    def __init__(self, streams: int, mixer_norm, mixer, ffn_norm=None, ffn=None, mixer_gate=None, ffn_gate=None, names=None):
        if not 1 <= streams <= ops.MAX_STREAMS:
            raise ValueError(f"{streams} streams (1 to {ops.MAX_STREAMS})")
        if ffn is None and (ffn_norm is not None or ffn_gate is not None):
            raise ValueError("a layer without a feed-forward has no norm or gate for it")
        self.streams = streams
        self.mixer_norm, self.mixer, self.mixer_gate, self.mixer_hyper = mixer_norm, mixer, mixer_gate, Hyper(streams)
        self.ffn_norm, self.ffn, self.ffn_gate = ffn_norm, ffn, ffn_gate
        self.ffn_hyper = Hyper(streams) if ffn is not None else None
        self.names = {"mixer_norm": "norm1", "mixer": "mix", "mixer_gate": "rg1", "mixer_hyper": "hc1",
                      "ffn_norm": "norm2", "ffn": "mlp", "ffn_gate": "rg2", "ffn_hyper": "hc2"}
        self.names.update(names or {})
        self._in = {}           # sublayer -> (stacked matrix, bias or None, columns of the gate)

    def _parts(self, prefix):
        for key in ("mixer_norm", "mixer", "mixer_gate", "mixer_hyper", "ffn_norm", "ffn", "ffn_gate", "ffn_hyper"):
            part = getattr(self, key)
            if part is not None:
                yield part, f"{prefix}.{self.names[key]}"

    def tensor_specs(self, prefix):
        return [s for part, p in self._parts(prefix) for s in part.tensor_specs(p)]

    def bind(self, prefix, tensors, rt):
        for part, p in self._parts(prefix):
            part.bind(p, tensors, rt)
        for key, sub, gate in (("mixer", self.mixer, self.mixer_gate), ("ffn", self.ffn, self.ffn_gate)):
            if sub is None:
                continue
            rows = getattr(sub, "in_rows", None)
            w, b = rows() if rows is not None else (None, None)
            mats, vecs = ([gate.w], [gate.b]) if gate is not None else ([], [])
            if w is not None:
                mats.append(w)
                vecs.append(b if b is not None else torch.zeros(w.shape[0], dtype=torch.float32, device=w.device))
            if mats:
                self._in[key] = (torch.cat(mats, dim=0).contiguous(), torch.cat(vecs).contiguous(), gate.w.shape[0] if gate is not None else 0)
                if gate is not None:
                    gate.w = None       # the stacked copy is what runs

    def cache_spec(self):
        return self.mixer.cache_spec()

    @property
    def graph_safe(self):
        return all(getattr(part, "graph_safe", False) for part, _ in self._parts(""))

    def _sublayer(self, rt, key, sub, h, *where):
        """(the sublayer's result, its gate's logits or None)."""
        stacked = self._in.get(key)
        if stacked is None:
            return sub.forward(rt, h, *where), None
        w, b, n_gate = stacked
        proj = rt.linear(h, w, bias=b, out_dtype=torch.float32)
        gate = proj[:, :n_gate] if n_gate else None
        if w.shape[0] == n_gate:
            return sub.forward(rt, h, *where), gate
        own = proj[:, n_gate:]
        return (sub.forward_projected(rt, own, *where) if key == "mixer" else sub.forward_projected(rt, h, own)), gate

    def forward(self, rt, x, pending, batch, cache):
        h = self.mixer_norm.forward(rt, x, rt.dtype, delta=pending, w_in=self.mixer_hyper.w_in)
        if self.ffn is not None:
            stacked = self._in.get("ffn")
            rt.ahead([stacked[0]] if stacked is not None else self.ffn.first_weights())       # read after the mixer: L2 may fetch it meanwhile
        y, gate = self._sublayer(rt, "mixer", self.mixer, h, batch, cache)
        pending = PendingStreams(delta=y, gate=gate, w_out=self.mixer_hyper.w_out, mix=self.mixer_hyper.mix)
        if self.ffn is not None:
            h = self.ffn_norm.forward(rt, x, rt.dtype, delta=pending, w_in=self.ffn_hyper.w_in)
            y, gate = self._sublayer(rt, "ffn", self.ffn, h)
            pending = PendingStreams(delta=y, gate=gate, w_out=self.ffn_hyper.w_out, mix=self.ffn_hyper.mix)
        return x, pending


register_part("norm", "stream_rmsnorm", StreamNorm)
register_part("block", "hyper", HyperBlock)
