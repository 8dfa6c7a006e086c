"""Pelenex's configuration: a decoder whose layers are listed one by one in config.json.

    {"architecture": "Pelenex", "vocab": …, "width": …, "norm": {"eps": …, "groups": …}, "logit_softcap": …,
     "layers": [{"type": "mlstm" | "parallel" | "channel_delta", "mixer": {…}, "mlp": {…} | null}, …]}

A layer names its mixer's kind and sizes and its feed-forward.

  "mlstm"          heads, dim, vdim, gate_cap
  "channel_delta"  heads, kv_heads, dim, vdim, conv (taps of the short convolution)
  "parallel"       left: heads, kv_heads, dim, vdim, scale, mask (size, keep_first); right: heads, dim, vdim, tau

A feed-forward is "dense" (`ff`) or "moe" (`expert.ff`, `router.experts`, `router.top`, `shared.ff`).  `norm.groups` (1),
`logit_softcap` (none), a mask (every earlier key is visible) and its `keep_first` (0), `mlp` and `shared` may each be
absent.
"""
from __future__ import annotations

import dataclasses

from .base import ConfigError, ModelConfig, key
from .kuvusun import _need

MIXER_TYPES = ("mlstm", "parallel", "channel_delta")
MLP_KINDS = ("dense", "moe")


@dataclasses.dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0                      # 0: every earlier key is visible
    keep_first: int = 0


@dataclasses.dataclass(frozen=True)
class MemoryConfig:
    heads: int
    dim: int
    vdim: int
    kv_heads: int = 0                    # channel_delta: query/key heads
    conv: int = 0                        # channel_delta: taps
    gate_cap: float = 0.0                # mlstm
    tau: float = 0.0                     # the right branch of "parallel"


@dataclasses.dataclass(frozen=True)
class MixerConfig:
    kind: str
    memory: MemoryConfig
    attention: AttentionConfig | None = None     # the left branch of "parallel"


@dataclasses.dataclass(frozen=True)
class FeedForwardConfig:
    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    shared_ff: int = 0                   # 0: no shared expert


@dataclasses.dataclass
class PelenexConfig(ModelConfig):
    model_type = "Pelenex"

    vocab: int = key()
    width: int = key()
    norm: dict = key()
    layers: list = key()
    logit_softcap: float = key(default=None, nullable=True)

    def to_dict(self) -> dict:
        out = {"architecture": self.model_type, "vocab": self.vocab, "width": self.width, "norm": self.norm, "layers": self.layers}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out

    def validate(self) -> None:
        self._positive("vocab", self.vocab)
        self._positive("width", self.width)
        self.norm_eps = _need(self.norm, "eps", float, "norm")
        self.norm_groups = _need(self.norm, "groups", int, "norm") if "groups" in self.norm else 1
        if not self.norm_eps > 0.0:
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps}")
        if self.norm_groups < 1 or self.width % self.norm_groups != 0:
            raise ConfigError(f"norm.groups ({self.norm_groups}) must cut the width ({self.width}) into equal parts")
        if self.logit_softcap is not None and not self.logit_softcap > 0.0:
            raise ConfigError(f"logit_softcap must be positive, got {self.logit_softcap}")
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        self.mixers = [self._mixer(i, layer) for i, layer in enumerate(self.layers)]
        self.mlps = [self._mlp(i, layer) for i, layer in enumerate(self.layers)]

    def _mixer(self, i: int, layer) -> MixerConfig:
        where = f"layers[{i}]"
        kind = _need(layer, "type", str, where)
        if kind not in MIXER_TYPES:
            raise ConfigError(f"config.json: {where}.type '{kind}' is not one of {', '.join(MIXER_TYPES)}")
        m = _need(layer, "mixer", dict, where)
        mw = where + ".mixer"
        if kind == "parallel":
            left, right = _need(m, "left", dict, mw), _need(m, "right", dict, mw)
            return MixerConfig(kind, self._memory(right, mw + ".right", tau=_need(right, "tau", float, mw + ".right")),
                               self._attention(left, mw + ".left"))
        if kind == "mlstm":
            return MixerConfig(kind, self._memory(m, mw, gate_cap=_need(m, "gate_cap", float, mw)))
        mc = self._memory(m, mw, kv_heads=_need(m, "kv_heads", int, mw), conv=_need(m, "conv", int, mw))
        if mc.heads % mc.kv_heads != 0:
            raise ConfigError(f"config.json: {mw}: kv_heads ({mc.kv_heads}) must divide heads ({mc.heads})")
        return MixerConfig(kind, mc)

    @staticmethod
    def _memory(m: dict, mw: str, **more) -> MemoryConfig:
        mc = MemoryConfig(_need(m, "heads", int, mw), _need(m, "dim", int, mw), _need(m, "vdim", int, mw), **more)
        for name, v in (("heads", mc.heads), ("dim", mc.dim), ("vdim", mc.vdim), *more.items()):
            if not v > 0:
                raise ConfigError(f"config.json: {mw}.{name} must be positive, got {v}")
        return mc

    @staticmethod
    def _attention(m: dict, mw: str) -> AttentionConfig:
        window = keep = 0
        mask = m.get("mask")
        if mask is not None:
            window = _need(mask, "size", int, mw + ".mask")
            if mask.get("keep_first") is not None:
                keep = _need(mask, "keep_first", int, mw + ".mask")
            if window <= 0 or keep < 0:
                raise ConfigError(f"config.json: {mw}.mask: size must be positive and keep_first not negative")
        ac = AttentionConfig(_need(m, "heads", int, mw), _need(m, "kv_heads", int, mw), _need(m, "dim", int, mw), _need(m, "vdim", int, mw),
                             _need(m, "scale", float, mw), window, keep)
        if min(ac.heads, ac.kv_heads, ac.dim, ac.vdim) <= 0 or ac.heads % ac.kv_heads != 0:
            raise ConfigError(f"config.json: {mw}: heads, kv_heads, dim and vdim must be positive and kv_heads divide heads")
        if ac.vdim != ac.dim:
            raise ConfigError(f"config.json: {mw}: the values of this mixer are its keys, so vdim ({ac.vdim}) must equal dim ({ac.dim})")
        return ac

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
            expert, router, shared = _need(ml, "expert", dict, lw), _need(ml, "router", dict, lw), ml.get("shared")
            cfg = FeedForwardConfig("moe", _need(expert, "ff", int, lw + ".expert"), experts=_need(router, "experts", int, lw + ".router"),
                                    top=_need(router, "top", int, lw + ".router"),
                                    shared_ff=_need(shared, "ff", int, lw + ".shared") if shared is not None else 0)
            if cfg.experts <= 0 or not (0 < cfg.top <= cfg.experts):
                raise ConfigError(f"config.json: {lw}.router: top ({cfg.top}) must lie in 1…experts ({cfg.experts})")
            if shared is not None and cfg.shared_ff <= 0:
                raise ConfigError(f"config.json: {lw}.shared.ff must be positive")
        if cfg.ff <= 0:
            raise ConfigError(f"config.json: {lw}: the inner size must be positive")
        return cfg

    @property
    def n_layer(self) -> int:
        return len(self.layers)
