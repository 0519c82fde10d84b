"""Typed configuration of the Zufotar design, read from its own config.json keys.

A Zufotar model is a list of layers whose mixer and feed-forward run side by side, each behind a norm of its own of the
same stream: x <- x + (mixer(norm1(x)) + ff(norm2(x))). A layer's mixer is one of two kinds. `latent_attention`: attention
over a cached latent per token, the queries out of a latent of their own, a rotated part with optionally scaled
frequencies (the yarn rule), an output gate as wide as the heads. `wkv`: a recurrence with decays per token and channel and
a bonus for the current token, behind a token shift. The feed-forward is dense with the erf form of gelu, a mixture of
gated experts (sigmoid scores, a correction for the choice, limited groups, optionally a gated shared expert), or absent.
A stretch of layers may run several times with the same weights; every pass begins with a learned vector added to the
stream, and every pass but the first with the embedding's output added before that. Logits are bounded. config.json gives
every size and every constant that can differ between models; nothing here assumes a value. Keys:

    architecture            "Zufotar"
    vocab, width            sizes of the embedding table (also the output matrix)
    embedding.scale         factor on the embedded rows
    norm.eps                eps of every RMS norm
    logit_softcap           bound of the logits; absent or null: none
    layers[i].type          "latent_attention" or "wkv"
    layers[i].mixer         latent_attention: {heads, dim, rot_dim, vdim, q_rank, kv_rank, scale,
                                rot {base, dims; optionally scaling {factor, original, fast, slow}}}
                            wkv: {heads, dim; optionally decay_rank, which a checkpoint's tensors give otherwise}
    layers[i].mlp           null, {kind "dense", ff}, or {kind "moe", expert {ff}, router {experts, top, scale,
                            groups {count, keep} or absent}, shared {ff} or absent}
    loop                    absent/null, or {start, stop, times}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .base import ConfigError, ModelConfig, looped_runs, read_eos, read_loop, require_float, require_int
from .base import require_object as _obj
from .danonex import YarnScaling


@dataclass(frozen=True)
class QueryLatentAttentionConfig:
    heads: int
    dim: int                 # unrotated query/key dimensions per head
    rot_dim: int             # rotated query/key dimensions per head (the key's are shared by all heads)
    vdim: int
    q_rank: int              # size of the queries' latent
    kv_rank: int             # size of the cached latent
    scale: float             # factor on the scores
    rot_base: float = 10000.0
    rot_dims: int = 0        # how many of the rot_dim dimensions are rotated
    rot_scaling: YarnScaling | None = None

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "QueryLatentAttentionConfig":
        rot = _obj(m, "rot", where, optional=True)
        base, dims, scaling = 10000.0, 0, None
        if rot is not None:
            base, dims = require_float(rot, "base"), require_int(rot, "dims", minimum=0)
            if base <= 0:
                raise ConfigError(f"{where}.rot: 'base' must be above 0, got {base}")
            s = _obj(rot, "scaling", where + ".rot", optional=True)
            if s is not None:
                scaling = YarnScaling.from_dict(s, where + ".rot.scaling")
                if base == 1.0:
                    raise ConfigError(f"{where}.rot: a base of 1 has no frequencies to scale")
        c = cls(require_int(m, "heads"), require_int(m, "dim"), require_int(m, "rot_dim", minimum=0), require_int(m, "vdim"),
                require_int(m, "q_rank"), require_int(m, "kv_rank"), require_float(m, "scale"), base, dims, scaling)
        if c.rot_dims > c.rot_dim or c.rot_dims % 2:
            raise ConfigError(f"{where}: rot.dims {c.rot_dims} must be even and at most rot_dim {c.rot_dim}")
        return c

    def to_dict(self) -> dict:
        rot: dict[str, Any] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.rot_scaling is not None:
            rot["scaling"] = self.rot_scaling.to_dict()
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                "kv_rank": self.kv_rank, "scale": self.scale, "rot": rot}


@dataclass(frozen=True)
class TimeMixingConfig:
    heads: int
    dim: int                         # key channels and value columns per head
    decay_rank: int | None = None    # rows of the decay's first projection; None: the checkpoint's tensor says

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "TimeMixingConfig":
        return cls(require_int(m, "heads"), require_int(m, "dim"),
                   None if m.get("decay_rank") is None else require_int(m, "decay_rank"))

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "dim": self.dim}
        if self.decay_rank is not None:
            d["decay_rank"] = self.decay_rank
        return d


@dataclass(frozen=True)
class ZufotarMLP:
    kind: str                        # "dense" or "moe"
    ff: int                          # inner size, of one expert for "moe"
    experts: int = 0
    top: int = 0
    scale: float = 1.0               # factor on the experts' weights
    groups: int = 1                  # experts form `groups` equal groups of neighbours
    keep: int = 1                    # only experts of the best `keep` groups can be chosen
    shared_ff: int | None = None     # inner size of the shared expert; None: there is none

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "ZufotarMLP":
        kind = m.get("kind")
        if kind == "dense":
            return cls("dense", require_int(m, "ff"))
        if kind != "moe":
            raise ConfigError(f"{where}: feed-forward kind {kind!r} is not known (known: 'dense', 'moe')")
        router = _obj(m, "router", where)
        groups = _obj(router, "groups", where + ".router", optional=True)
        shared = _obj(m, "shared", where, optional=True)
        c = cls("moe", require_int(_obj(m, "expert", where), "ff"), require_int(router, "experts"), require_int(router, "top"),
                require_float(router, "scale", default=1.0), 1 if groups is None else require_int(groups, "count"),
                1 if groups is None else require_int(groups, "keep"), None if shared is None else require_int(shared, "ff"))
        if c.experts % c.groups or c.keep > c.groups:
            raise ConfigError(f"{where}: {c.experts} experts do not form {c.groups} equal groups of which {c.keep} are kept")
        if c.top > c.experts // c.groups * c.keep:
            raise ConfigError(f"{where}: top {c.top} exceeds the experts of the kept groups")
        return c

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        r: dict[str, Any] = {"experts": self.experts, "top": self.top, "scale": self.scale}
        if self.groups > 1:
            r["groups"] = {"count": self.groups, "keep": self.keep}
        d: dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff}, "router": r}
        if self.shared_ff is not None:
            d["shared"] = {"ff": self.shared_ff}
        return d


MIXER_CONFIGS = {"latent_attention": QueryLatentAttentionConfig, "wkv": TimeMixingConfig}


@dataclass(frozen=True)
class ZufotarLayer:
    type: str
    mixer: Any
    mlp: ZufotarMLP | None


@dataclass(frozen=True)
class ZufotarConfig(ModelConfig):
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    layers: tuple
    logit_softcap: float | None = None
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1      # layers loop_start .. loop_stop-1 run this many times in a row
    eos_token_ids: tuple = ()

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "ZufotarConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(L, dict) or L.get("type") not in MIXER_CONFIGS:
                raise ConfigError(f"{where}: 'type' must be one of {sorted(MIXER_CONFIGS)}, got "
                                  f"{L.get('type') if isinstance(L, dict) else L!r}")
            mlp = _obj(L, "mlp", where, optional=True)
            layers.append(ZufotarLayer(L["type"], MIXER_CONFIGS[L["type"]].from_dict(_obj(L, "mixer", where), where + ".mixer"),
                                       None if mlp is None else ZufotarMLP.from_dict(mlp, where + ".mlp")))
        softcap = None if raw.get("logit_softcap") is None else require_float(raw, "logit_softcap")
        if softcap is not None and softcap <= 0:
            raise ConfigError(f"config.json: 'logit_softcap' must be above 0, got {softcap}")
        return cls(require_int(raw, "vocab"), require_int(raw, "width"),
                   require_float(_obj(raw, "embedding", "config.json"), "scale"),
                   require_float(_obj(raw, "norm", "config.json"), "eps"), tuple(layers), softcap,
                   *read_loop(raw, len(layers)), read_eos(raw))

    @property
    def has_loop(self) -> bool:
        return self.loop_stop > self.loop_start

    def layer_runs(self) -> list[tuple[int, int | None]]:
        """[(layer, pass number if the run begins a pass of the loop, else None)] in running order."""
        return looped_runs(len(self.layers), self.loop_start, self.loop_stop, self.loop_times)

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {
            "architecture": "Zufotar", "vocab": self.vocab, "width": self.width,
            "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
            "layers": [{"type": L.type, "mixer": L.mixer.to_dict(), "mlp": None if L.mlp is None else L.mlp.to_dict()}
                       for L in self.layers]}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.has_loop:
            d["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
