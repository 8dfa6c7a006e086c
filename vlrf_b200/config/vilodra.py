"""Vilodra's configuration: a decoder whose layers are listed one by one in config.json.

    {"architecture": "Vilodra", "vocab": …, "width": …, "norm": {"eps": …}, "residual_mult": …,
     "layers": [{"type": "attention" | "latent_attention" | "lightning", "mixer": {…}, "mlp": {…} | null}, …]}

A layer names its mixer's kind and sizes and its feed-forward.

  "attention"         heads, kv_heads, dim (of one of a head's two maps), vdim, scale, diff, rot (base, dims, scaling: factor,
                      low, high, original)
  "latent_attention"  heads, dim, rot_dim, vdim, kv_rank, scale, mask (size), rot (base, dims, scaling: factor, original, fast,
                      slow), kv_from (an earlier layer of this kind whose latents this one reads)
  "lightning"         heads, dim, vdim, decay (one number per head)

A feed-forward is "dense" (`ff`) or "moe" (`expert.ff`, `router.experts`, `router.top`, `router.scale`).  `residual_mult` (1), a
mixer's `rot` ("attention"), `rot.scaling`, `mask` (every earlier key is visible), `kv_from`, and `mlp` may each be absent.
"""
from __future__ import annotations

import dataclasses

from .base import ConfigError, ModelConfig, key
from .kuvusun import _need

MIXER_TYPES = ("attention", "latent_attention", "lightning")
MLP_KINDS = ("dense", "moe")


@dataclasses.dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int
    #: "attention": (factor, low, high, original); "latent_attention": (factor, original, fast, slow); None: unscaled
    scaling: tuple | None = None


@dataclasses.dataclass(frozen=True)
class DifferentialConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: RotationConfig | None = None
    kind = "attention"


@dataclasses.dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: RotationConfig
    window: int = 0                      # 0: every earlier key is visible
    kv_from: int | None = None
    kind = "latent_attention"


@dataclasses.dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple
    kind = "lightning"


@dataclasses.dataclass(frozen=True)
class FeedForwardConfig:
    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    scale: float = 1.0


def _rotation(m: dict, mw: str, names: tuple):
    rot = m.get("rot")
    if rot is None:
        return None
    rw = mw + ".rot"
    scaling = rot.get("scaling") if isinstance(rot, dict) else None
    if scaling is not None:
        scaling = tuple(_need(scaling, name, float, rw + ".scaling") for name in names)
        if min(scaling) <= 0.0:
            raise ConfigError(f"config.json: {rw}.scaling: {', '.join(names)} must be positive")
    out = RotationConfig(_need(rot, "base", float, rw), _need(rot, "dims", int, rw), scaling)
    if out.dims <= 0 or out.dims % 2 != 0 or not out.base > 0.0:
        raise ConfigError(f"config.json: {rw}: dims ({out.dims}) must be even and positive, and base positive")
    return out


@dataclasses.dataclass
class VilodraConfig(ModelConfig):
    model_type = "Vilodra"

    vocab: int = key()
    width: int = key()
    norm: dict = key()
    layers: list = key()
    residual_mult: float = key(default=1.0)

    def to_dict(self) -> dict:
        return {"architecture": self.model_type, "vocab": self.vocab, "width": self.width, "norm": self.norm,
                "residual_mult": self.residual_mult, "layers": self.layers}

    def validate(self) -> None:
        self._positive("vocab", self.vocab)
        self._positive("width", self.width)
        self.norm_eps = _need(self.norm, "eps", float, "norm")
        if not self.norm_eps > 0.0:
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps}")
        self.residual_mult = float(self.residual_mult)
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        self.mixers, self.mlps = [], []
        for i, layer in enumerate(self.layers):
            self.mixers.append(self._mixer(i, layer))
            self.mlps.append(self._mlp(i, layer))

    def _mixer(self, i: int, layer):
        where = f"layers[{i}]"
        kind = _need(layer, "type", str, where)
        if kind not in MIXER_TYPES:
            raise ConfigError(f"config.json: {where}.type '{kind}' is not one of {', '.join(MIXER_TYPES)}")
        m = _need(layer, "mixer", dict, where)
        mw = where + ".mixer"

        def sizes(*names):
            out = {name: _need(m, name, int, mw) for name in names}
            for name, v in out.items():
                if v <= 0:
                    raise ConfigError(f"config.json: {mw}.{name} must be positive, got {v}")
            return out
        if kind == "lightning":
            n = sizes("heads", "dim", "vdim")
            decay = _need(m, "decay", list, mw)
            if not isinstance(decay, list) or len(decay) != n["heads"] \
                    or any(isinstance(a, bool) or not isinstance(a, (int, float)) for a in decay):
                raise ConfigError(f"config.json: {mw}.decay must hold one number per head ({n['heads']})")
            return LightningConfig(decay=tuple(float(a) for a in decay), **n)
        if kind == "attention":
            mc = DifferentialConfig(scale=_need(m, "scale", float, mw), diff=_need(m, "diff", float, mw),
                                    rot=_rotation(m, mw, ("factor", "low", "high", "original")), **sizes("heads", "kv_heads", "dim", "vdim"))
            if mc.heads % mc.kv_heads != 0:
                raise ConfigError(f"config.json: {mw}: kv_heads ({mc.kv_heads}) must divide heads ({mc.heads})")
            if mc.rot is not None and mc.rot.dims > mc.dim:
                raise ConfigError(f"config.json: {mw}: rot.dims ({mc.rot.dims}) must be at most dim ({mc.dim})")
            if mc.rot is not None and mc.rot.scaling is not None and not mc.rot.scaling[1] < mc.rot.scaling[2]:
                raise ConfigError(f"config.json: {mw}.rot.scaling: low must be below high")
            return mc
        rot = _rotation(m, mw, ("factor", "original", "fast", "slow"))
        if rot is None:
            raise ConfigError(f"config.json: {mw} lacks 'rot'")
        window = 0
        if m.get("mask") is not None:
            window = _need(m["mask"], "size", int, mw + ".mask")
            if window <= 0:
                raise ConfigError(f"config.json: {mw}.mask.size must be positive, got {window}")
        mc = LatentConfig(scale=_need(m, "scale", float, mw), rot=rot, window=window,
                          kv_from=_need(m, "kv_from", int, mw) if m.get("kv_from") is not None else None,
                          **sizes("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        if rot.dims > mc.rot_dim:
            raise ConfigError(f"config.json: {mw}: rot.dims ({rot.dims}) must be at most rot_dim ({mc.rot_dim})")
        if rot.scaling is not None and rot.base == 1.0:
            raise ConfigError(f"config.json: {mw}.rot: a base of 1 cannot be scaled")
        if mc.kv_from is not None:
            j = mc.kv_from
            if not (0 <= j < i) or self.mixers[j].kind != "latent_attention" or self.mixers[j].kv_from is not None:
                raise ConfigError(f"config.json: {mw}.kv_from = {j} must name an earlier layer of the same kind with latents of its own")
            o = self.mixers[j]
            if (o.kv_rank, o.rot_dim, o.rot) != (mc.kv_rank, mc.rot_dim, mc.rot):
                raise ConfigError(f"config.json: {mw}: kv_rank, rot_dim and rot differ from those of layer {j}, whose latents it reads")
        return mc

    @staticmethod
    def _mlp(i: int, layer):
        ml = layer.get("mlp") if isinstance(layer, dict) else None
        if ml is None:
            return None
        lw = f"layers[{i}].mlp"
        mk = _need(ml, "kind", str, lw)
        if mk not in MLP_KINDS:
            raise ConfigError(f"config.json: {lw}.kind '{mk}' is not one of {', '.join(MLP_KINDS)}")
        if mk == "dense":
            cfg = FeedForwardConfig("dense", _need(ml, "ff", int, lw))
        else:
            expert, router, rw = _need(ml, "expert", dict, lw), _need(ml, "router", dict, lw), lw + ".router"
            cfg = FeedForwardConfig("moe", _need(expert, "ff", int, lw + ".expert"), experts=_need(router, "experts", int, rw),
                                    top=_need(router, "top", int, rw), scale=_need(router, "scale", float, rw))
            if cfg.experts <= 0 or not (0 < cfg.top <= cfg.experts):
                raise ConfigError(f"config.json: {rw}: top ({cfg.top}) must lie in 1…experts ({cfg.experts})")
        if cfg.ff <= 0:
            raise ConfigError(f"config.json: {lw}: the inner size must be positive")
        return cfg

    def cache_window(self, i: int) -> int:
        """How many of the latest rows the cache that layer i reads must keep (0: all): the widest window of the layers that
        read it."""
        owner = self.mixers[i].kv_from if self.mixers[i].kv_from is not None else i
        windows = [m.window for k, m in enumerate(self.mixers)
                   if m.kind == "latent_attention" and (k == owner or m.kv_from == owner)]
        return 0 if 0 in windows else max(windows)

    @property
    def n_layer(self) -> int:
        return len(self.layers)
