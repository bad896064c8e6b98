"""Kadodra as a model description: a decoder-only design whose layers are listed one by one in config.json.  A layer is
``x + (mixer(h) + ff(h))`` with ONE RMS norm ``h = norm1(x)`` feeding both sublayers.  Its mixer is a latent attention
(parts/latent.py: queries straight from the input, a rotate-half rotation with rescaled frequencies, a sliding window, a
learned sink per head) or lightning attention (parts/retention.py: linear attention with a fixed decay per head, the
activations of q, k and v a silu, one norm over all heads and a sigmoid gate).  The feed-forward is dense with the square
of relu or a mixture of experts that a table indexed by the token's id chooses, the experts' gate and up clipped.  A range
of layers may run several times in a row, every pass with caches and states of its own and the embedding output added to
the residual ahead of every pass but the first.  The output matrix is the embedding table and the logits are scaled.

Tensor names: ``embed``, ``final.norm``; layer i: ``l<i>.norm1``; latent attention ``l<i>.mix.{q,dkv,dkv.norm,uk,uv,sink,
o}``; lightning ``l<i>.mix.{q,k,v,g,o,norm}``; dense ``l<i>.mlp.{up,down}``; experts ``l<i>.mlp.table`` and
``l<i>.mlp.e<j>.{gate,up,down}``."""
from __future__ import annotations

from ..config.kadodra_config import KadodraConfig
from ..parts.description import ModelDescription, LayerSpec, PartSpec, ScheduleEntry
from ..registry import register_architecture

ARCHITECTURE = "Kadodra"


def describe_kadodra(cfg: KadodraConfig) -> ModelDescription:
    W = cfg.hidden_size
    positions, layers = {}, []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}"
        position = None
        if l.latent is not None:
            a = l.latent
            position = f"halves:{a.rot.dims}:{a.rot.base!r}:{a.rot.scaling!r}"
            if position not in positions:
                positions[position] = PartSpec("scaled_rotary", dict(rotary_dim=a.rot.dims, theta=a.rot.base,
                                                                     pairing="halves", scaling=a.rot.scaling))
            mixer = PartSpec("latent_attention", dict(
                hidden_size=W, num_heads=a.heads, head_dim=a.dim, rot_dim=a.rot_dim, v_head_dim=a.vdim, q_rank=0,
                kv_rank=a.kv_rank, eps=cfg.norm_eps, softmax_scale=a.scale, window=a.window, sink=True), prefix=f"{p}.mix")
        else:
            r = l.lightning
            mixer = PartSpec("lightning_attention", dict(
                hidden_size=W, num_heads=r.heads, head_dim=r.dim, v_head_dim=r.vdim, decay=r.decay, eps=cfg.norm_eps),
                prefix=f"{p}.mix")
        ff = None
        if l.mlp is not None and l.mlp.kind == "dense":
            ff = PartSpec("plain_mlp", dict(hidden_size=W, intermediate_size=l.mlp.ff, activation="relu2"), prefix=f"{p}.mlp")
        elif l.mlp is not None:
            ff = PartSpec("routed_experts", dict(
                hidden_size=W, intermediate_size=l.mlp.ff, num_experts=l.mlp.experts, top=l.mlp.top,
                activation="clipped_swish", activation_limit=l.mlp.limit, router_score="table", table_rows=cfg.vocab_size,
                weight_on="output"), prefix=f"{p}.mlp")
        layers.append(LayerSpec(mixer=mixer, feed_forward=ff, block="parallel_shared_norm", position=position,
                                mixer_norm=PartSpec("rms_norm", dict(dim=W, eps=cfg.norm_eps, name="norm1"), prefix=p)))
    return ModelDescription(
        hidden_size=W, vocab_size=cfg.vocab_size, max_position=cfg.max_position, embed_name="embed", lm_head_name=None,
        final_norm=PartSpec("rms_norm", dict(dim=W, eps=cfg.norm_eps, name="norm"), prefix="final"),
        layers=layers, schedule=[ScheduleEntry(layer=i, add_embedding=again) for i, again in cfg.runs()],
        positions=positions, logit_scale=cfg.logit_scale)


register_architecture(ARCHITECTURE, KadodraConfig.from_json_dict, describe_kadodra, replace=True)
