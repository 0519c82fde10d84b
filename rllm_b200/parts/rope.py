"""Rotary position encoding as a part: a table of inverse frequencies, made once on the
host in float64 and kept as float32; the rotation itself runs inside the kernel that
also writes K and V to the cache.

Plain rule f_i = theta^(-2i/d): src/gpu/cuda/shaders/rope.cu:62-66 of the reference. A
model's own rule (`rope_scaling.rope_type`) is looked up by name in `rope_rules`.
"""
from __future__ import annotations

import torch

from .base import Part, register_part
from .rope_rules import rope_magnitude, rope_rule


def _rule_params(rot_dim, theta, scaling) -> dict:
    return dict(scaling.to_dict(), base=float(theta), dims=rot_dim)


def table_magnitude(rot_dim: int, theta: float, scaling=None) -> float:
    """The factor a scaling rule puts on every cosine and sine (1 without one)."""
    if scaling is None or scaling.rope_type == "default":
        return 1.0
    return rope_magnitude(scaling.rope_type, _rule_params(rot_dim, theta, scaling))


def inverse_frequencies(rot_dim: int, theta: float, scaling=None) -> list[float]:
    """The rot_dim/2 inverse frequencies in float64, the scaling rule applied. `scaling`: None, or
    an object with `rope_type` and `to_dict()` (the rule's parameters)."""
    freqs = [float(theta) ** (-2.0 * i / rot_dim) for i in range(rot_dim // 2)]
    if scaling is not None and scaling.rope_type != "default":
        freqs = list(rope_rule(scaling.rope_type)(freqs, _rule_params(rot_dim, theta, scaling)))
        if len(freqs) != rot_dim // 2:
            raise ValueError(f"rope rule {scaling.rope_type!r} returned {len(freqs)} frequencies for {rot_dim // 2}")
    return freqs


class RotaryEmbedding(Part):
    """Rotates pairs (i, i + rot_dim/2) of each head by position * f_i."""
    graph_safe = True
    interleaved = False

    def __init__(self, head_dim: int, theta: float, scaling=None, rot_dim: int | None = None):
        self.head_dim = head_dim
        self.rot_dim = head_dim if rot_dim is None else rot_dim
        if self.rot_dim % 2 or self.rot_dim > head_dim:
            raise ValueError(f"rotary width {self.rot_dim} must be even and <= head_dim {head_dim}")
        self.theta, self.scaling = float(theta), scaling
        self.inv_freq = None
        # layers with the same rule share one table of angles per step
        self.table_key = ("rope", self.rot_dim, self.theta, repr(scaling))

    def finalize(self, device, dtype):
        f = inverse_frequencies(self.rot_dim, self.theta, self.scaling)
        self.inv_freq = torch.tensor(f, dtype=torch.float64).to(torch.float32).to(device)
        self.mag = table_magnitude(self.rot_dim, self.theta, self.scaling)

    @property
    def rotated(self) -> int:
        """How many leading dimensions of a head turn."""
        return self.rot_dim

    def table(self, ctx):
        """float32 [T, rot_dim/2, 2] (cos, sin) for the step's tokens, shared by the layers of one rule."""
        return ctx.backend.rope_table(ctx, ctx.positions, self.inv_freq, self.rot_dim, self.table_key, self.mag)

    def project_rotate_store(self, x, w_qkv, bias, ctx, cache, nh, nkv):
        """qkv = x w_qkv^T (+ bias) with q and k rotated and k, v written into the layer's pages:
        the projection and this part's work in one kernel where the backend can."""
        if self.mag != 1.0:
            self.table(ctx)            # the backend finds the step's table, made with the factor, by its key
        return ctx.backend.qkv_rope_cache_write(x, w_qkv, bias, ctx.positions, self.inv_freq, cache, nh, nkv,
                                                self.head_dim, self.rot_dim, ctx=ctx, key=self.table_key)

    def rotate_and_store(self, qkv, ctx, cache, nh, nkv):
        """Rotate q (in place) and k of `qkv`, and write k, v into the layer's pages."""
        if self.mag != 1.0:
            self.table(ctx)
        ctx.backend.rope_cache_write(qkv, ctx.positions, self.inv_freq, cache, nh, nkv,
                                     self.head_dim, self.rot_dim, ctx=ctx, key=self.table_key)


class InterleavedRotary(Part):
    """Rotates pairs (2i, 2i+1), i < dims/2, of a vector of `rot_dim` numbers by position * f_i with
    f_i = base^(-2i/dims); the dimensions from `dims` on pass unchanged. The part owns the rule (the
    frequencies and the step's table of cos and sin); the rotation itself runs inside the kernel of
    the mixer that uses it. `scaling`: a rule of `rope_rules` on the frequencies (and, for rules that have one, a factor
    on all cosines and sines)."""
    graph_safe = True
    interleaved = True

    def __init__(self, rot_dim: int, base: float, dims: int | None = None, scaling=None):
        self.rot_dim = rot_dim
        self.dims = rot_dim if dims is None else dims
        if self.dims % 2 or self.dims > rot_dim:
            raise ValueError(f"rotated dimensions {self.dims} must be even and <= {rot_dim}")
        self.base, self.scaling = float(base), scaling
        self.inv_freq = None
        self.table_key = ("rope_interleaved", self.dims, self.base, repr(scaling))

    def finalize(self, device, dtype):
        f = inverse_frequencies(self.dims, self.base, self.scaling)
        self.inv_freq = torch.tensor(f, dtype=torch.float64).to(torch.float32).to(device)
        self.mag = table_magnitude(self.dims, self.base, self.scaling)

    @property
    def rotated(self) -> int:
        return self.dims

    def table(self, ctx):
        """float32 [T, dims/2, 2] (cos, sin) for the step's tokens, shared by the layers of one rule."""
        if self.dims == 0:
            return torch.empty((ctx.num_tokens, 0, 2), dtype=torch.float32, device=self.inv_freq.device)
        return ctx.backend.rope_table(ctx, ctx.positions, self.inv_freq, self.dims, self.table_key, self.mag)


register_part("position", "rope", RotaryEmbedding)
register_part("position", "rope_interleaved", InterleavedRotary)
