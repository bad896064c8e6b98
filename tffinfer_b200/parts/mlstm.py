"""The matrix memory of xLSTM (mLSTM): linear attention over a matrix state per head with an input gate and a forget gate per
head and token that are exponentials, held in range by a running maximum, and a normaliser that follows the keys.

For head h with queries and keys of ``head_dim`` (K) and values of ``v_head_dim`` (V) elements:

    q_t = W_q x_t * K^-1/2      k_t = W_k x_t      v_t = W_v x_t
    i_t = cap tanh((W_i x_t + b_i) / cap)          f_t = logsigmoid(cap tanh((W_f x_t + b_f) / cap))
    m_t = max(f_t + m_(t-1), i_t)                  the running maximum, 0 ahead of the request's first token
    S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T          S [K, V] and n [K] start from zeros
    n_t = e^(f_t + m_(t-1) - m_t) n_(t-1) + e^(i_t - m_t) k_t
    o_t = S_t^T q_t / (max(|n_t . q_t|, e^-m_t) + 1e-6)
    out = W_o( concat_h( o_t / rms(o_t) ) * w * sigmoid(W_g x_t) )           rms over the head's V elements with ``eps``

The projections are one product; its float32 accumulators go to the recurrence, whose gates, decays, normaliser and state are
float32 in either mode of the engine.  The state is a ``StateNeed``: a slot holds the heads' S, then their n, then their m."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..registry import register_part
from .base import Mixer, SplitMixer, WeightSpec, MATRIX, VECTOR, StateNeed, LayerContext


@register_part("mixer", "mlstm")
class MLstm(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, v_head_dim: int, gate_cap: float, eps: float,
                 names: Optional[Dict[str, str]] = None, prefix: str = ""):
        super().__init__(prefix)
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.head_dim, self.v_head_dim = int(head_dim), int(v_head_dim)
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        if min(self.num_heads, self.head_dim, self.v_head_dim) <= 0 or not self.gate_cap > 0 or not self.eps > 0:
            raise ValueError("mlstm: heads, sizes, gate_cap and eps must be positive")
        self.names = {"q": "q", "k": "k", "v": "v", "gate": "g", "o": "o", "norm": "norm", "in": "i", "in_bias": "i.b",
                      "forget": "f", "forget_bias": "f.b"}
        self.names.update(names or {})
        self.qk_width, self.v_width = self.num_heads * self.head_dim, self.num_heads * self.v_head_dim
        self.w_in = self.w_o = self.norm_w = self.gate_bias = None

    def kernel_files(self):
        return ("mlstm", "gated_norm")

    def cache_need(self):
        from ..kernels.library import mlstm_state_size
        return StateNeed((mlstm_state_size(self.num_heads, self.head_dim, self.v_head_dim),), "float32", self_starting=True)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        n, H, W = self.names, self.num_heads, self.hidden_size
        return {n["q"]: WeightSpec((self.qk_width, W), MATRIX), n["k"]: WeightSpec((self.qk_width, W), MATRIX),
                n["v"]: WeightSpec((self.v_width, W), MATRIX), n["gate"]: WeightSpec((self.v_width, W), MATRIX),
                n["o"]: WeightSpec((W, self.v_width), MATRIX),
                n["norm"]: WeightSpec((self.v_width,), VECTOR, init="one_plus_normal"),
                n["in"]: WeightSpec((H, W), MATRIX), n["in_bias"]: WeightSpec((H,), VECTOR, init="normal", init_scale=1.0),
                n["forget"]: WeightSpec((H, W), MATRIX),
                n["forget_bias"]: WeightSpec((H,), VECTOR, init="one_plus_normal", init_scale=1.0)}

    def load(self, tensors, ops, act_dtype) -> None:
        n = self.names
        rows = [tensors[n[w]] for w in ("q", "k", "v", "gate", "in", "forget")]
        dt = rows[0].dtype if all(r.dtype == rows[0].dtype for r in rows) else torch.float32
        self.w_in = SplitMixer.padded_rows(torch.cat([r.to(dt) for r in rows], dim=0))
        self.w_o = tensors[n["o"]]
        self.norm_w = tensors[n["norm"]].to(torch.float32).contiguous()
        self.gate_bias = torch.cat([tensors[n["in_bias"]].to(torch.float32), tensors[n["forget_bias"]].to(torch.float32)]).contiguous()

    takes_projection = True

    def forward(self, h, ctx: LayerContext, residual, proj=None):
        if ctx.state is None:
            raise ValueError("mlstm needs a state tensor (StateNeed)")
        ops = ctx.ops
        T = h.shape[0]
        mixed = torch.empty((T, self.v_width), dtype=h.dtype, device=h.device)
        ops.mlstm(h, self.w_in, ctx.batch, ctx.state, self.gate_bias, self.gate_cap, self.norm_w, self.eps, mixed,
                  self.num_heads, self.head_dim, self.v_head_dim, proj=proj)
        if residual is None:
            out = ops.sublayer_output(T, self.hidden_size, h.device, h.dtype, self.output_use)
            ops.gemm(mixed, self.w_o, out)
            return out
        ops.gemm(mixed, self.w_o, residual, residual=residual)
        return residual
