"""Gumodra as a model description: a decoder-only design whose layers are listed one by one in config.json.  A layer is
``x + mixer(h) s(R1 h + b1) + ff(h) s(R2 h + b2)`` (s the sigmoid) with ONE RMS norm ``h = norm1(x)``, whose weight is a single
number, feeding both sublayers and both gates.  Its mixer is a grouped-query attention (parts/attention.py: biases, per-head
norms of q and k, a rotate-half rotation, values that are the keys as projected, a window beside the kept first tokens, a
learned sink per head) or a matrix memory with exponential gates (parts/mlstm.py).  The feed-forward is dense or a mixture of
experts chosen within groups, beside a shared expert behind a gate of its own (parts/moe.py).  The embedding is scaled; the
output matrix is a tensor of its own.

Tensor names: ``embed``, ``head``, ``final.norm``; layer i: ``l<i>.norm1``, ``l<i>.{rg1,rg2}`` with ``.b``; attention
``l<i>.mix.{q,k,o}`` with ``.b``, ``l<i>.mix.{q.norm,k.norm,sink}``; mlstm ``l<i>.mix.{q,k,v,g,o,norm,i,i.b,f,f.b}``; dense
``l<i>.mlp.{gate,up,down}``; experts ``l<i>.mlp.{router,correction}``, ``l<i>.mlp.e<j>.{gate,up,down}`` and
``l<i>.mlp.shared.{gate,up,down,sg}``."""
from __future__ import annotations

from ..config.gumodra_config import GumodraConfig
from ..parts.description import ModelDescription, LayerSpec, PartSpec, ScheduleEntry
from ..registry import register_architecture

ARCHITECTURE = "Gumodra"


def describe_gumodra(cfg: GumodraConfig) -> ModelDescription:
    W = cfg.hidden_size
    positions, layers = {}, []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}"
        position = None
        if l.attention is not None:
            a = l.attention
            if a.rot is not None:
                position = f"halves:{a.rot.dims}:{a.rot.base!r}"
                positions.setdefault(position, PartSpec("scaled_rotary", dict(rotary_dim=a.rot.dims, theta=a.rot.base,
                                                                              pairing="halves")))
            mixer = PartSpec("gated_sink_attention", dict(
                hidden_size=W, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, softmax_scale=a.scale,
                window=a.window, keep_first=a.keep_first, sink="learned", qk_norm="head", qk_norm_eps=cfg.norm_eps,
                projection_bias=True, values_are_keys=True,
                names={"q": "q", "k": "k", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "sink": "sink",
                       "q_bias": "q.b", "k_bias": "k.b", "o_bias": "o.b"}), prefix=f"{p}.mix")
        else:
            r = l.mlstm
            mixer = PartSpec("mlstm", dict(hidden_size=W, num_heads=r.heads, head_dim=r.dim, v_head_dim=r.vdim,
                                           gate_cap=r.gate_cap, eps=cfg.norm_eps), prefix=f"{p}.mix")
        ff = None
        if l.mlp is not None and l.mlp.kind == "dense":
            ff = PartSpec("swiglu", dict(hidden_size=W, intermediate_size=l.mlp.ff, activation="silu",
                                         names={"gate": "gate", "up": "up", "down": "down"}), prefix=f"{p}.mlp")
        elif l.mlp is not None:
            ff = PartSpec("routed_experts", dict(
                hidden_size=W, intermediate_size=l.mlp.ff, num_experts=l.mlp.experts, top=l.mlp.top, activation="silu",
                renormalize=True, weight_on="output", router_score="softmax", correction=True, groups=l.mlp.groups,
                shared_intermediate=l.mlp.shared_ff, shared_gate=l.mlp.shared_ff > 0), prefix=f"{p}.mlp")
        layers.append(LayerSpec(
            mixer=mixer, feed_forward=ff, block="gated_parallel", position=position,
            mixer_norm=PartSpec("rms_norm", dict(dim=W, eps=cfg.norm_eps, name="norm1", one_number=True), prefix=p),
            connectors={"gates": PartSpec("residual_gates", dict(hidden_size=W, feed_forward=ff is not None), prefix=p)}))
    return ModelDescription(
        hidden_size=W, vocab_size=cfg.vocab_size, max_position=cfg.max_position, embed_name="embed", lm_head_name="head",
        final_norm=PartSpec("rms_norm", dict(dim=W, eps=cfg.norm_eps, name="norm", one_number=True), prefix="final"),
        layers=layers, schedule=[ScheduleEntry(layer=i) for i in range(len(layers))], positions=positions,
        embed_scale=cfg.embed_scale, streams=1)


register_architecture(ARCHITECTURE, GumodraConfig.from_json_dict, describe_gumodra, replace=True)
