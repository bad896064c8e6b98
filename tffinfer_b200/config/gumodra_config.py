"""Typed configuration of the Gumodra design: a decoder-only model whose config.json lists its layers one by one.  A layer
is one RMS norm (with a single number for a weight) whose output feeds a mixer and a feed-forward side by side; what each of
them gives is multiplied, element by element, by a sigmoid gate read from the same input before it joins the residual.  The
mixer is ``attention`` (grouped-query attention whose values are its keys as projected, a sliding window beside the kept
first tokens, a learned sink per head) or ``mlstm`` (a matrix memory with exponential gates and a running maximum); the
feed-forward is dense, a mixture of experts chosen within groups beside a gated shared expert, or absent.

    {"architecture": "Gumodra", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size", "keep_first"},
                           "rot": {"base", "dims"}},
                 "mlp": {"kind": "dense", "ff": F}
                        | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "groups": {"count", "keep"}},
                           "shared": {"ff"}}
                        | null},
                {"type": "mlstm", "mixer": {"heads", "dim", "vdim", "gate_cap"}, "mlp": ...}, ...]}

Every size and constant of a checkpoint comes from there.  Optional keys: ``embedding.scale`` (absent: 1), ``kv_heads``
(absent: heads), ``vdim`` of an attention (absent: dim; the values are the keys, so it can be nothing else), ``mask``
(absent: all earlier keys), ``mask.keep_first`` (absent: none), ``rot`` (absent: no rotation), ``groups`` (absent: one
group), ``shared`` (absent: no shared expert), ``max_position`` (absent: MAX_POSITION_DEFAULT; the design itself has no
limit, the engine's block tables need one)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .model_config import ModelConfig, ConfigError
from .tipezen_config import RotaryConfig, _need, _int, _float, MAX_POSITION_DEFAULT


@dataclass(frozen=True)
class GumodraMlp:
    kind: str                          # "dense" | "moe"
    ff: int
    experts: int = 0
    top: int = 0
    groups: Tuple[int, int] = (1, 1)   # count of groups, groups kept
    shared_ff: int = 0                 # 0 = no shared expert


@dataclass(frozen=True)
class GumodraAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot: Optional[RotaryConfig] = None
    window: int = 0                    # 0 = all earlier keys
    keep_first: int = 0


@dataclass(frozen=True)
class GumodraMlstm:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class GumodraLayer:
    type: str                          # "attention" | "mlstm"
    attention: Optional[GumodraAttention] = None
    mlstm: Optional[GumodraMlstm] = None
    mlp: Optional[GumodraMlp] = None


def _read_mlp(mlp, where: str) -> Optional[GumodraMlp]:
    if mlp is None:
        return None
    kind = _need(mlp, "kind", where)
    if kind == "dense":
        out = GumodraMlp("dense", _int(mlp, "ff", where))
    elif kind == "moe":
        e, r = _need(mlp, "expert", where), _need(mlp, "router", where)
        g, s = r.get("groups"), mlp.get("shared")
        groups = (1, 1) if g is None else (_int(g, "count", where + ".router.groups"), _int(g, "keep", where + ".router.groups"))
        out = GumodraMlp("moe", _int(e, "ff", where + ".expert"), _int(r, "experts", where + ".router"),
                         _int(r, "top", where + ".router"), groups, 0 if s is None else _int(s, "ff", where + ".shared"))
        if not 0 < out.top <= out.experts:
            raise ConfigError(f"config.json: {where}.router: 1 <= top <= experts, got top {out.top} of {out.experts}")
        count, keep = groups
        if count < 1 or not 1 <= keep <= count or out.experts % count or out.top > keep * (out.experts // count):
            raise ConfigError(f"config.json: {where}.router.groups: {count} groups of which {keep} are kept must divide "
                              f"{out.experts} experts evenly and leave at least top ({out.top}) of them")
        if s is not None and out.shared_ff <= 0:
            raise ConfigError(f"config.json: {where}.shared: 'ff' must be positive")
    else:
        raise ConfigError(f"config.json: {where}.kind '{kind}' is not a feed-forward of this design (dense, moe)")
    if out.ff <= 0:
        raise ConfigError(f"config.json: {where}: 'ff' must be positive")
    return out


def _read_attention(m, where: str) -> GumodraAttention:
    heads, dim = _int(m, "heads", where), _int(m, "dim", where)
    mask, window, keep = m.get("mask"), 0, 0
    if mask is not None:
        window, keep = _int(mask, "size", where + ".mask"), _int(mask, "keep_first", where + ".mask", 0)
        if window <= 0 or keep < 0:
            raise ConfigError(f"config.json: {where}.mask: 'size' must be positive and 'keep_first' not negative")
    out = GumodraAttention(heads=heads, kv_heads=_int(m, "kv_heads", where, heads), dim=dim, scale=_float(m, "scale", where),
                           rot=RotaryConfig.read(m.get("rot"), where + ".rot"), window=window, keep_first=keep)
    if min(out.heads, out.kv_heads, out.dim) <= 0 or out.heads % out.kv_heads:
        raise ConfigError(f"config.json: {where}: heads, kv_heads and dim must be positive and heads a multiple of kv_heads")
    if _int(m, "vdim", where, dim) != dim:
        raise ConfigError(f"config.json: {where}: the values are the keys, so 'vdim' must be 'dim' ({dim})")
    if out.rot is not None and out.rot.dims > dim:
        raise ConfigError(f"config.json: {where}.rot: 'dims' ({out.rot.dims}) must be at most dim ({dim})")
    if out.rot is not None and out.rot.scaling is not None:
        raise ConfigError(f"config.json: {where}.rot: this design does not rescale its frequencies")
    return out


def _read_mlstm(m, where: str) -> GumodraMlstm:
    out = GumodraMlstm(heads=_int(m, "heads", where), dim=_int(m, "dim", where), vdim=_int(m, "vdim", where),
                       gate_cap=_float(m, "gate_cap", where))
    if min(out.heads, out.dim, out.vdim) <= 0 or not out.gate_cap > 0:
        raise ConfigError(f"config.json: {where}: heads, dim, vdim and gate_cap must be positive")
    return out


@dataclass(frozen=True)
class GumodraConfig(ModelConfig):
    vocab_size: int = 0
    hidden_size: int = 0
    norm_eps: float = 0.0
    embed_scale: float = 1.0
    layers: Tuple[GumodraLayer, ...] = ()
    max_position: int = MAX_POSITION_DEFAULT

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @staticmethod
    def from_json_dict(d: Dict[str, Any]) -> "GumodraConfig":
        from .model_config import architecture_name
        raw = _need(d, "layers", "the top level")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, l in enumerate(raw):
            where = f"layers[{i}]"
            kind = _need(l, "type", where)
            m = _need(l, "mixer", where)
            mlp = _read_mlp(l.get("mlp"), where + ".mlp")
            if kind == "attention":
                layers.append(GumodraLayer(kind, attention=_read_attention(m, where + ".mixer"), mlp=mlp))
            elif kind == "mlstm":
                layers.append(GumodraLayer(kind, mlstm=_read_mlstm(m, where + ".mixer"), mlp=mlp))
            else:
                raise ConfigError(f"config.json: {where}.type '{kind}' is not a mixer of this design (attention, mlstm)")
        cfg = GumodraConfig(
            architecture=architecture_name(d), vocab_size=_int(d, "vocab", "the top level"),
            hidden_size=_int(d, "width", "the top level"), norm_eps=_float(_need(d, "norm", "the top level"), "eps", "norm"),
            embed_scale=_float(d.get("embedding") or {}, "scale", "embedding", 1.0), layers=tuple(layers),
            max_position=_int(d, "max_position", "the top level", MAX_POSITION_DEFAULT))
        if cfg.vocab_size <= 0 or cfg.hidden_size <= 0 or not cfg.norm_eps > 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive and norm.eps > 0")
        return cfg

    def to_json_dict(self) -> Dict[str, Any]:
        out = []
        for l in self.layers:
            m: Dict[str, Any]
            if l.attention is not None:
                a = l.attention
                m = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.dim, "scale": a.scale}
                if a.rot is not None:
                    m["rot"] = a.rot.to_json()
                if a.window > 0:
                    m["mask"] = {"size": a.window, "keep_first": a.keep_first}
            else:
                r = l.mlstm
                m = {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "gate_cap": r.gate_cap}
            mlp: Optional[Dict[str, Any]] = None
            if l.mlp is not None and l.mlp.kind == "dense":
                mlp = {"kind": "dense", "ff": l.mlp.ff}
            elif l.mlp is not None:
                router: Dict[str, Any] = {"experts": l.mlp.experts, "top": l.mlp.top}
                if l.mlp.groups != (1, 1):
                    router["groups"] = {"count": l.mlp.groups[0], "keep": l.mlp.groups[1]}
                mlp = {"kind": "moe", "expert": {"ff": l.mlp.ff}, "router": router}
                if l.mlp.shared_ff > 0:
                    mlp["shared"] = {"ff": l.mlp.shared_ff}
            out.append({"type": l.type, "mixer": m, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                             "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embed_scale}, "layers": out}
        if self.max_position != MAX_POSITION_DEFAULT:
            d["max_position"] = self.max_position
        return d
