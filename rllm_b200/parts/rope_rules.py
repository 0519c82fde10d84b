"""Rules that turn the plain rotary frequencies f_i = theta^(-2i/d) into a model's own, by name.

A rule is a function `(inverse frequencies as float64 list, the rule's parameters as a dict) ->
list` (the dict also holds the rotation's `base` and `dims`) and, optionally, a check of the parameters that
raises ValueError and a factor on all cosines and sines. The name is what a
config.json carries in `rope_scaling.rope_type`; the configuration reader accepts exactly the
registered names and the rotary part applies the rule, so another rule (another family's long
context scheme) is one `register_rope_rule` call, from anywhere.

Built in: "linear" (every frequency divided by `factor`), "yarn" (slow frequencies divided by `factor`, fast ones kept,
a ramp over the index between, and a factor on cosines and sines that grows with ln `factor`) and "llama3", the three bands of the
reference's "yarn" kernel (src/gpu/cuda/shaders/rope.cu:233-251) with beta_fast =
high_freq_factor and beta_slow = low_freq_factor. The reference parses `rope_scaling` for Llama
(src/model/config.rs:724-746) but never applies it; here it is applied.
"""
from __future__ import annotations

import math
from typing import Callable

_RULES: dict[str, tuple[Callable, Callable | None, Callable | None]] = {}


def register_rope_rule(name: str, rule: Callable[[list[float], dict], list[float]],
                       check: Callable[[dict], None] | None = None,
                       magnitude: Callable[[dict], float] | None = None) -> None:
    """`magnitude`: a function of the rule's parameters that gives the factor on every cosine and sine (None: 1)."""
    _RULES[name] = (rule, check, magnitude)


def registered_rope_rules() -> list[str]:
    return sorted(_RULES)


def rope_rule(name: str) -> Callable[[list[float], dict], list[float]]:
    try:
        return _RULES[name][0]
    except KeyError:
        raise KeyError(f"no rotary frequency rule named {name!r}; registered: {registered_rope_rules()}") from None


def rope_magnitude(name: str, params: dict) -> float:
    """The factor a rule puts on every cosine and sine."""
    rule = _RULES.get(name)
    return 1.0 if rule is None or rule[2] is None else float(rule[2](params))


def check_rope_rule(name: str, params: dict) -> None:
    """Raise ValueError if the rule's parameters are missing or out of range."""
    rule = _RULES.get(name)
    if rule is None:
        raise ValueError(f"rope_scaling.rope_type {name!r} is not supported (supported: "
                         f"{['default'] + registered_rope_rules()})")
    if rule[1] is not None:
        rule[1](params)


def _need(params: dict, key: str, kind=float):
    v = params.get(key)
    if v is None:
        raise ValueError(f"config.json lacks required key {key!r} (in rope_scaling)")
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (kind is int and not isinstance(v, int)):
        raise ValueError(f"config key {key!r} (in rope_scaling) must be a number, got {v!r}")
    return v


def _linear(freqs, p):
    return [f / float(p["factor"]) for f in freqs]


def _check_factor(p):
    if _need(p, "factor") <= 0:
        raise ValueError(f"rope_scaling.factor must be > 0, got {p['factor']}")


def _llama3(freqs, p):
    factor, low, high = float(p["factor"]), float(p.get("low_freq_factor", 1.0)), float(p.get("high_freq_factor", 4.0))
    orig = float(p["original_max_position_embeddings"])
    out = []
    for f in freqs:
        wavelen = 2.0 * math.pi / f
        if wavelen < orig / high:
            pass
        elif wavelen > orig / low:
            f = f / factor
        else:
            s = (orig / wavelen - low) / (high - low)
            f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def _check_llama3(p):
    _check_factor(p)
    low = p.get("low_freq_factor", 1.0)
    high = p.get("high_freq_factor", 4.0)
    if _need(p, "original_max_position_embeddings", int) < 1:
        raise ValueError("rope_scaling.original_max_position_embeddings must be >= 1")
    if high <= low:
        raise ValueError(f"rope_scaling: high_freq_factor must exceed low_freq_factor (got low={low}, high={high})")


def _yarn(freqs, p):
    """Frequency i turns original * f_i / (2 pi) times over the original context. Up to the index where that is `fast`
    turns frequencies stay, from the index where it is `slow` on they are divided by `factor`, linear in the index
    between; both indices are rounded outwards and kept inside 0 .. dims - 1."""
    dims, base, factor = int(p["dims"]), float(p["base"]), float(p["factor"])

    def index(turns):
        return dims * math.log(float(p["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index(float(p["fast"]))), 0)
    hi = min(math.ceil(index(float(p["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out


def _check_yarn(p):
    for key in ("factor", "original", "fast", "slow"):
        v = p.get(key)
        if isinstance(v, bool) or not isinstance(v, (int, float)) or v <= 0:
            raise ValueError(f"yarn scaling of the rotation: {key!r} must be a number above 0, got {v!r}")


def _yarn_magnitude(p):
    return 0.1 * math.log(float(p["factor"])) + 1.0


register_rope_rule("linear", _linear, _check_factor)
register_rope_rule("yarn", _yarn, _check_yarn, _yarn_magnitude)
register_rope_rule("llama3", _llama3, _check_llama3)
