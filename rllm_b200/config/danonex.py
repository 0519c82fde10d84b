"""Typed configuration of the Danonex design, read from its own config.json keys.

A Danonex model is a list of layers that norm what a sublayer gives, not what it reads: x <- x + m * norm1(mixer(x)), then
x <- x + m * norm2(ff(x)) (a layer may have no feed-forward), m one number for the model. A layer's mixer is one of two
kinds. `delta`: a gated delta rule, queries, keys and values each behind a short causal convolution, one decay and one
step size per head, an output gate. `attention`: grouped-query attention whose queries and keys are normed over all
heads together, an interleaved rotation of part of each head (its frequencies optionally scaled by the yarn rule), bounded
scores and a sink. The feed-forward is W_down gelu(W_up x) with the erf form of gelu. The output matrix is the
embedding table, logits are multiplied by a number. config.json gives every size and every constant that can differ
between models; nothing here assumes a value. Keys:

    architecture            "Danonex"
    vocab, width            sizes of the embedding table (also the output matrix)
    norm.eps                eps of every RMS norm
    residual_mult           m
    logit_scale             factor on the logits
    layers[i].type          "delta" or "attention"
    layers[i].mixer         delta: {heads, kv_heads, dim, vdim, conv}
                            attention: {heads, kv_heads, dim, vdim, scale; optionally softcap,
                                        rot {base, dims; optionally scaling {factor, original, fast, slow}}}
    layers[i].mlp           null, or {kind "dense", ff}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .base import ConfigError, ModelConfig, require_float, require_int


def _obj(raw: dict, key: str, where: str, optional: bool = False):
    v = raw.get(key)
    if v is None:
        if optional:
            return None
        raise ConfigError(f"{where} lacks required key {key!r}")
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: {key!r} must be an object, got {v!r}")
    return v


def _heads(m: dict, where: str):
    heads, kv = require_int(m, "heads"), require_int(m, "kv_heads")
    if heads % kv:
        raise ConfigError(f"{where}: {heads} heads do not divide over {kv} kv_heads")
    return heads, kv


def _positive(m: dict, key: str, where: str) -> float:
    v = require_float(m, key)
    if v <= 0:
        raise ConfigError(f"{where}: {key!r} must be above 0, got {v}")
    return v


@dataclass(frozen=True)
class YarnScaling:
    """Parameters of the rotation rule "yarn" (`parts.rope_rules`), under this design's key names."""
    factor: float
    original: float               # positions of the context the frequencies were made for
    fast: float                   # turns over it from which on a frequency is kept
    slow: float                   # turns over it up to which a frequency is divided by `factor`
    rope_type = "yarn"

    @classmethod
    def from_dict(cls, s: dict, where: str) -> "YarnScaling":
        return cls(*(_positive(s, key, where) for key in ("factor", "original", "fast", "slow")))

    def to_dict(self) -> dict:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class HeadDecayDeltaConfig:
    heads: int
    kv_heads: int
    dim: int                      # query/key size per head
    vdim: int                     # value size per head
    conv: int                     # taps of the short convolutions

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "HeadDecayDeltaConfig":
        heads, kv = _heads(m, where)
        return cls(heads, kv, require_int(m, "dim"), require_int(m, "vdim"), require_int(m, "conv"))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}


@dataclass(frozen=True)
class BoundedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float                      # factor on the scores
    softcap: float | None = None      # bound of the scores; None: not bounded
    rot_dims: int = 0                 # leading dimensions of a head that are rotated; 0: no rotation
    rot_base: float = 10000.0
    rot_scaling: YarnScaling | None = None

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "BoundedAttentionConfig":
        heads, kv = _heads(m, where)
        rot = _obj(m, "rot", where, optional=True)
        dims, base, scaling = 0, 10000.0, None
        if rot is not None:
            dims, base = require_int(rot, "dims", minimum=0), _positive(rot, "base", where + ".rot")
            s = _obj(rot, "scaling", where + ".rot", optional=True)
            if s is not None:
                scaling = YarnScaling.from_dict(s, where + ".rot.scaling")
                if base == 1.0:
                    raise ConfigError(f"{where}.rot: a base of 1 has no frequencies to scale")
        softcap = None if m.get("softcap") is None else _positive(m, "softcap", where)
        c = cls(heads, kv, require_int(m, "dim"), require_int(m, "vdim"), require_float(m, "scale"), softcap, dims, base, scaling)
        if c.rot_dims % 2 or c.rot_dims > c.dim:
            raise ConfigError(f"{where}.rot: {c.rot_dims} rotated dimensions must be even and at most dim {c.dim}")
        return c

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale}
        if self.softcap is not None:
            d["softcap"] = self.softcap
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_scaling is not None:
                d["rot"]["scaling"] = self.rot_scaling.to_dict()
        return d


MIXER_CONFIGS = {"delta": HeadDecayDeltaConfig, "attention": BoundedAttentionConfig}


@dataclass(frozen=True)
class DanonexLayer:
    type: str
    mixer: Any
    ff: int | None                # inner size of the dense feed-forward; None: the layer has none


@dataclass(frozen=True)
class DanonexConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_scale: float
    layers: tuple
    eos_token_ids: tuple = ()

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "DanonexConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(L, dict) or L.get("type") not in MIXER_CONFIGS:
                raise ConfigError(f"{where}: 'type' must be one of {sorted(MIXER_CONFIGS)}, got "
                                  f"{L.get('type') if isinstance(L, dict) else L!r}")
            mixer = MIXER_CONFIGS[L["type"]].from_dict(_obj(L, "mixer", where), where + ".mixer")
            mlp = L.get("mlp")
            ff = None
            if mlp is not None:
                if not isinstance(mlp, dict):
                    raise ConfigError(f"{where}: 'mlp' must be an object or null")
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"{where}.mlp: feed-forward kind {mlp.get('kind')!r} is not known (known: 'dense')")
                ff = require_int(mlp, "ff")
            layers.append(DanonexLayer(L["type"], mixer, ff))
        eos = raw.get("eos_token_id")
        eos = () if eos is None else tuple(eos) if isinstance(eos, (list, tuple)) else (eos,)
        return cls(require_int(raw, "vocab"), require_int(raw, "width"),
                   require_float(_obj(raw, "norm", "config.json"), "eps"), require_float(raw, "residual_mult"),
                   require_float(raw, "logit_scale"), tuple(layers), tuple(int(e) for e in eos))

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {
            "architecture": "Danonex", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult, "logit_scale": self.logit_scale,
            "layers": [{"type": L.type, "mixer": L.mixer.to_dict(),
                        "mlp": None if L.ff is None else {"kind": "dense", "ff": L.ff}} for L in self.layers]}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
