"""A gated residual: a sublayer's result is multiplied, element by element, by a sigmoid read from the sublayer's own input
before it joins the residual, and the arrangement of two sublayers side by side over it:

    h = norm(x)
    x <- x + mixer(h) * sigmoid(R1 h + b1) + feed_forward(h) * sigmoid(R2 h + b2)

R1 and R2 are [hidden, hidden] and run as one product (tensors "rg1", "rg1.b", "rg2", "rg2.b" unless ``names`` says
otherwise).  The sum is float32; both sublayers' outputs, their gates and the next layer's norm meet in one kernel
(``ops.gated_join``, csrc/streams.cu), which runs when the residual is read again."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..registry import register_part
from .base import Block, Connector, LayerContext, WeightSpec, MATRIX, VECTOR
from .streams import ResidualStreams


@register_part("connector", "residual_gates")
class ResidualGates(Connector):
    """The gates of a layer's mixer and (``feed_forward``) of its feed-forward."""

    def __init__(self, hidden_size: int, feed_forward: bool = True, names: Optional[Dict[str, str]] = None, prefix: str = ""):
        super().__init__(prefix)
        self.hidden_size, self.feed_forward = int(hidden_size), bool(feed_forward)
        self.names = {"mixer": "rg1", "mixer_bias": "rg1.b", "ffn": "rg2", "ffn_bias": "rg2.b"}
        self.names.update(names or {})
        self.w = self.bias = self.w_all = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        n, W = self.names, self.hidden_size
        s = {n["mixer"]: WeightSpec((W, W), MATRIX), n["mixer_bias"]: WeightSpec((W,), VECTOR, init="normal", init_scale=0.5)}
        # a layer of a mixer alone may still carry the second pair in a file: it is accepted and not used
        s[n["ffn"]] = WeightSpec((W, W), MATRIX, optional=not self.feed_forward)
        s[n["ffn_bias"]] = WeightSpec((W,), VECTOR, init="normal", init_scale=0.5, optional=not self.feed_forward)
        return s

    def load(self, tensors, ops, act_dtype) -> None:
        n = self.names
        rows = [tensors[n["mixer"]]] + ([tensors[n["ffn"]]] if self.feed_forward else [])
        bias = [tensors[n["mixer_bias"]]] + ([tensors[n["ffn_bias"]]] if self.feed_forward else [])
        dt = rows[0].dtype if all(r.dtype == rows[0].dtype for r in rows) else torch.float32
        self.w = torch.cat([r.to(dt) for r in rows], dim=0).contiguous()
        self.bias = torch.cat([b.to(torch.float32) for b in bias]).contiguous()

    def share_rows(self, mixer) -> None:
        """Puts the rows of the mixer's input product and those of the gates side by side in one matrix, of which both keep
        their part: where few tokens make every product a pass over its weights, the two run as one."""
        if not getattr(mixer, "takes_projection", False) or mixer.w_in.dtype != self.w.dtype:
            return
        n = mixer.w_in.shape[0]
        self.w_all = torch.cat([mixer.w_in, self.w], dim=0).contiguous()
        mixer.w_in, self.w = self.w_all[:n], self.w_all[n:]

    def gates(self, h, ops) -> torch.Tensor:
        """The gates ahead of bias and sigmoid, [T, hidden] or [T, 2 * hidden]."""
        z = ops.gate_rows(h.shape[0], self.w.shape[0], h.device, h.dtype)
        ops.gemm(h, self.w, z)
        return z

    def read(self, x: ResidualStreams, norm, ops, out_dtype):
        return x.read(None, norm, ops, out_dtype)

    def write(self, x: ResidualStreams, y, z=None, mixer_bias=None, y_ff=None, gate_col: int = 0) -> None:
        x.write_gated(z, self.bias, y, mixer_bias, y_ff, gate_col)


@register_part("block", "gated_parallel")
class GatedParallelBlock(Block):
    """The mixer and the feed-forward side by side on ONE norm's output, each behind a gate of ``connectors["gates"]``; a
    layer without a feed-forward is the mixer alone."""

    def __init__(self, mixer, feed_forward=None, mixer_norm=None, ffn_norm=None, extra_norms=None, connectors=None):
        super().__init__(mixer, feed_forward, mixer_norm, ffn_norm, extra_norms, connectors)
        if mixer_norm is None or ffn_norm is not None or "gates" not in self.connectors:
            raise ValueError("the gated_parallel arrangement needs one norm, mixer_norm, and a 'gates' connector")
        mixer.output_use = "mixer behind a gate"           # both outputs wait for the kernel that joins them
        if feed_forward is not None:
            feed_forward.output_use = "feed-forward behind a gate"

    def loaded(self) -> None:
        self.connectors["gates"].share_rows(self.mixer)

    def forward(self, x: ResidualStreams, ctx: LayerContext, act_dtype):
        join, ops = self.connectors["gates"], ctx.ops
        h = join.read(x, self.mixer_norm, ops, act_dtype)
        if join.w_all is not None and ops.joins_products(h):        # one product for the mixer's input and the gates
            z, col = ops.projection_buffer(h.shape[0], join.w_all.shape[0], h.device, h.dtype, "with gates"), self.mixer.w_in.shape[0]
            ops.gemm(h, join.w_all, z)
            y = self.mixer.forward(h, ctx, residual=None, proj=z)
        else:
            z, col = join.gates(h, ops), 0
            y = self.mixer.forward(h, ctx, residual=None)
        f = self.feed_forward.forward(h, ctx, residual=None) if self.feed_forward is not None else None
        join.write(x, y, z, self.mixer.output_bias, f, col)
        return x
