"""Typed configuration of the Kadodra design: a decoder-only model whose config.json lists its layers one by one.  A
layer is one RMS norm whose output feeds a mixer and a feed-forward side by side; both are added to the residual.  The
mixer is ``latent_attention`` (windowed, with a learned sink per head, queries straight from the input) or ``lightning``
(linear attention with a fixed decay per head); the feed-forward is dense (the square of relu), a mixture of experts that
a table chooses by the token's id, or absent.  A range of layers may run several times in a row (``loop``), every pass
with caches and states of its own and the embedding output added to the residual ahead of it.

    {"architecture": "Kadodra", "vocab": V, "width": W, "norm": {"eps": e}, "logit_scale": s,
     "loop": {"start": i, "stop": j, "times": n},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "mask": {"size"},
                           "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}},
                 "mlp": {"kind": "dense", "ff": F} | {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"}}
                        | null},
                {"type": "lightning", "mixer": {"heads", "dim", "vdim", "decay": [...]}, "mlp": ...}, ...]}

Every size and constant of a checkpoint comes from there.  Optional keys: ``logit_scale`` (absent: 1), ``loop`` (absent:
every layer runs once), ``mask`` (absent: all earlier keys), ``rot.dims`` (absent: rot_dim), ``rot.scaling`` (absent:
plain frequencies), ``max_position`` (absent: MAX_POSITION_DEFAULT; the design itself has no limit, the engine's block
tables need one)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .model_config import ModelConfig, ConfigError
from .tipezen_config import RotaryConfig, _need, _int, _float, MAX_POSITION_DEFAULT


@dataclass(frozen=True)
class KadodraMlp:
    kind: str                          # "dense" | "moe"
    ff: int
    experts: int = 0
    top: int = 0
    limit: float = 0.0                 # bound of the experts' gate (above) and up (both sides)


@dataclass(frozen=True)
class KadodraLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: RotaryConfig
    window: int = 0                    # 0 = all earlier keys


@dataclass(frozen=True)
class KadodraLightning:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class KadodraLayer:
    type: str                          # "latent_attention" | "lightning"
    latent: Optional[KadodraLatent] = None
    lightning: Optional[KadodraLightning] = None
    mlp: Optional[KadodraMlp] = None


def _read_mlp(mlp, where: str) -> Optional[KadodraMlp]:
    if mlp is None:
        return None
    kind = _need(mlp, "kind", where)
    if kind == "dense":
        out = KadodraMlp("dense", _int(mlp, "ff", where))
    elif kind == "moe":
        e, r = _need(mlp, "expert", where), _need(mlp, "router", where)
        out = KadodraMlp("moe", _int(e, "ff", where + ".expert"), _int(r, "experts", where + ".router"),
                         _int(r, "top", where + ".router"), _float(e, "limit", where + ".expert"))
        if not 0 < out.top <= out.experts:
            raise ConfigError(f"config.json: {where}.router: 1 <= top <= experts, got top {out.top} of {out.experts}")
        if not out.limit > 0:
            raise ConfigError(f"config.json: {where}.expert: 'limit' must be positive")
    else:
        raise ConfigError(f"config.json: {where}.kind '{kind}' is not a feed-forward of this design (dense, moe)")
    if out.ff <= 0:
        raise ConfigError(f"config.json: {where}: 'ff' must be positive")
    return out


def _read_latent(m, where: str) -> KadodraLatent:
    rot_dim = _int(m, "rot_dim", where)
    raw = dict(_need(m, "rot", where))
    raw.setdefault("dims", rot_dim)
    mask = m.get("mask")
    window = 0
    if mask is not None:
        window = _int(mask, "size", where + ".mask")
        if window <= 0:
            raise ConfigError(f"config.json: {where}.mask: 'size' must be positive")
    out = KadodraLatent(
        heads=_int(m, "heads", where), dim=_int(m, "dim", where), rot_dim=rot_dim, vdim=_int(m, "vdim", where),
        kv_rank=_int(m, "kv_rank", where), scale=_float(m, "scale", where), rot=RotaryConfig.read(raw, where + ".rot"),
        window=window)
    if min(out.heads, out.dim, out.rot_dim, out.vdim, out.kv_rank) <= 0:
        raise ConfigError(f"config.json: {where}: heads, dim, rot_dim, vdim and kv_rank must be positive")
    if out.rot.dims > rot_dim:
        raise ConfigError(f"config.json: {where}.rot: 'dims' ({out.rot.dims}) must be at most rot_dim ({rot_dim})")
    if out.rot.scaling is not None and min(out.rot.scaling) <= 0:
        raise ConfigError(f"config.json: {where}.rot.scaling: every value must be positive")
    return out


def _read_lightning(m, where: str) -> KadodraLightning:
    decay = _need(m, "decay", where)
    if not isinstance(decay, list) or any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in decay):
        raise ConfigError(f"config.json: {where}: 'decay' must be a list of numbers")
    out = KadodraLightning(heads=_int(m, "heads", where), dim=_int(m, "dim", where), vdim=_int(m, "vdim", where),
                           decay=tuple(float(x) for x in decay))
    if min(out.heads, out.dim, out.vdim) <= 0:
        raise ConfigError(f"config.json: {where}: heads, dim and vdim must be positive")
    if len(out.decay) != out.heads:
        raise ConfigError(f"config.json: {where}: 'decay' lists {len(out.decay)} values for {out.heads} heads")
    return out


@dataclass(frozen=True)
class KadodraConfig(ModelConfig):
    vocab_size: int = 0
    hidden_size: int = 0
    norm_eps: float = 0.0
    logit_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None          # (start, stop, times)
    layers: Tuple[KadodraLayer, ...] = ()
    max_position: int = MAX_POSITION_DEFAULT

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def runs(self):
        """(layer, whether the embedding output is added to the residual ahead of it) in the order the layers run."""
        n = len(self.layers)
        start, stop, times = self.loop if self.loop is not None else (0, 0, 0)
        out = [(i, False) for i in range(start)]
        for t in range(times):
            out += [(i, t > 0 and i == start) for i in range(start, stop)]
        return out + [(i, False) for i in range(stop, n)]

    @staticmethod
    def from_json_dict(d: Dict[str, Any]) -> "KadodraConfig":
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
            if kind == "latent_attention":
                layers.append(KadodraLayer(kind, latent=_read_latent(m, where + ".mixer"), mlp=mlp))
            elif kind == "lightning":
                layers.append(KadodraLayer(kind, lightning=_read_lightning(m, where + ".mixer"), mlp=mlp))
            else:
                raise ConfigError(f"config.json: {where}.type '{kind}' is not a mixer of this design "
                                  f"(latent_attention, lightning)")
        loop = d.get("loop")
        lp = None
        if loop is not None:
            lp = (_int(loop, "start", "loop"), _int(loop, "stop", "loop"), _int(loop, "times", "loop"))
            if not 0 <= lp[0] < lp[1] <= len(layers) or lp[2] < 1:
                raise ConfigError(f"config.json: loop: 0 <= start < stop <= {len(layers)} layers and times >= 1, got {lp}")
        cfg = KadodraConfig(
            architecture=architecture_name(d), vocab_size=_int(d, "vocab", "the top level"),
            hidden_size=_int(d, "width", "the top level"), norm_eps=_float(_need(d, "norm", "the top level"), "eps", "norm"),
            logit_scale=_float(d, "logit_scale", "the top level", 1.0), loop=lp, layers=tuple(layers),
            max_position=_int(d, "max_position", "the top level", MAX_POSITION_DEFAULT))
        if cfg.vocab_size <= 0 or cfg.hidden_size <= 0 or not cfg.norm_eps > 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive and norm.eps > 0")
        return cfg

    def to_json_dict(self) -> Dict[str, Any]:
        out = []
        for l in self.layers:
            if l.latent is not None:
                a = l.latent
                m: Dict[str, Any] = {"heads": a.heads, "dim": a.dim, "rot_dim": a.rot_dim, "vdim": a.vdim,
                                     "kv_rank": a.kv_rank, "scale": a.scale, "rot": a.rot.to_json()}
                if a.window > 0:
                    m["mask"] = {"size": a.window}
            else:
                r = l.lightning
                m = {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay)}
            mlp: Optional[Dict[str, Any]] = None
            if l.mlp is not None and l.mlp.kind == "dense":
                mlp = {"kind": "dense", "ff": l.mlp.ff}
            elif l.mlp is not None:
                mlp = {"kind": "moe", "expert": {"ff": l.mlp.ff, "limit": l.mlp.limit},
                       "router": {"experts": l.mlp.experts, "top": l.mlp.top}}
            out.append({"type": l.type, "mixer": m, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                             "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale, "layers": out}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        if self.max_position != MAX_POSITION_DEFAULT:
            d["max_position"] = self.max_position
        return d
