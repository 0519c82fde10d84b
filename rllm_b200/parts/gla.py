"""Gated linear attention as a mixer part: a recurrence over a per-request state.

Per head, with h the mixer's input: q = W_q h * dim^-1/2, k = W_k h (`dim` key channels), v = W_v h
(`vdim`), a decay per key channel alpha = sigmoid(z)^(1/tau) with z = W_a2 (W_a1 h) + b, and
    S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,      o_t = S_t^T q_t.
Each head's o is RMS-normed over vdim with one weight of size vdim shared by the heads; the heads are
concatenated, multiplied by silu(W_g h) and projected by W_o. The state S starts at zero, is float32
and lives in a state slot of the cache manager (`StateSpec`), carried from step to step; decays,
the recurrence and the norm are float, the projections run in the run dtype. The width of the
decay's bottleneck (rows of W_a1) is a size of the checkpoint, not of the configuration: it is taken
from the tensor unless `decay_rank` is given (random-weights mode).

`TimeMixing` is the same kind of recurrence behind a token shift. With n the stream under the layer's norm and n' the
previous token's n (zeros for the first), five mixes x_s = n + (n' - n) * mu_s feed r, k, v, a gate and the decays; per
head (`dim` key channels and value columns)
    o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t,   S_t = diag(w_t) S_(t-1) + k_t v_t^T,   w = exp(-exp(W_w2 tanh(W_w1 x_w) + w0)),
so a token's own contribution is read with the bonus u in place of a decay. Each head's o is divided by its root mean
square; the heads, concatenated, are multiplied by a weight of their own, by silu of the gate, and projected by W_o. The
state is S and the last token's n, float. The mixer norms the stream itself (`norms_stream`): norm, shift and the five mixes are
one kernel.
"""
from __future__ import annotations

import torch

from .base import Param, Part, Source, StateSpec, register_part


def scan_chunk(ctx, chunk: int) -> int:
    """Long portions are cut into chunks that run side by side (the host knows a step's longest portion; inside a
    decode graph it is one token); 0: no chunks."""
    return chunk if not ctx.graph_safe and ctx.max_q_len >= 3 * chunk else 0


class GatedLinearAttention(Part):
    graph_safe = True
    takes_deferred = True
    returns_output = True

    def __init__(self, hidden: int, heads: int, dim: int, vdim: int, tau: float, eps: float = 1e-6,
                 decay_rank: int | None = None):
        self.hidden, self.heads, self.dim, self.vdim = hidden, heads, dim, vdim
        self.tau, self.eps, self.decay_rank = float(tau), float(eps), decay_rank
        self.chunk = 128         # tokens per chunk of a long portion
        self.w_in = self.w_a2 = self.b_a2 = self.w_norm = self.w_o = None

    def params(self):
        H, W, r = self.heads, self.hidden, -1 if self.decay_rank is None else self.decay_rank
        return [Param("w_in", (Source("q", (H * self.dim, W)), Source("k", (H * self.dim, W)),
                               Source("v", (H * self.vdim, W)), Source("g", (H * self.vdim, W)),
                               Source("a1", (r, W)))),
                Param("w_a2", (Source("a2", (H * self.dim, r)),)),
                Param("b_a2", (Source("a2.b", (H * self.dim,)),), role="vector"),
                Param("w_norm", (Source("norm", (self.vdim,), init="norm"),), role="vector"),
                Param("w_o", (Source("o", (W, H * self.vdim)),))]

    def cache_spec(self):
        return StateSpec((("S", (self.heads, self.dim, self.vdim), torch.float32),))

    def finalize(self, device, dtype):
        self._b_f32 = self.b_a2.float().contiguous()
        self._norm_f32 = self.w_norm.float().contiguous()
        self._a1_off = 2 * self.heads * (self.dim + self.vdim)
        if self.w_a2.shape[1] != self.w_in.shape[0] - self._a1_off:
            raise ValueError(f"{self.prefix}a1 has {self.w_in.shape[0] - self._a1_off} rows, a2 takes {self.w_a2.shape[1]}")

    def forward(self, x, ctx, cache, residual=None):
        be = ctx.backend
        H, d, v = self.heads, self.dim, self.vdim
        proj = be.linear(x, self.w_in)                                   # [T, q | k | v | gate | a1]
        z = be.linear_f32(proj[:, self._a1_off:], self.w_a2)             # float decay logits [T, H * dim]
        alpha = be.gla_decay(z, self._b_f32, self.tau)                   # in place
        o = be.gla_scan(proj, 0, H * d, 2 * H * d, alpha, d ** -0.5, H, d, v, ctx.cu_q, ctx.num_seqs,
                        ctx.state_slots, cache.state["S"], scan_chunk(ctx, self.chunk))
        att = be.gla_finish(o, self._norm_f32, self.eps, proj, 2 * H * d + H * v)
        if residual is None:
            return be.linear_f32(att, self.w_o)
        be.linear_residual(att, self.w_o, residual)
        return None


class TimeMixing(Part):
    graph_safe = True
    norms_stream = True
    returns_output = True
    SHIFTED = ("r", "k", "v", "g", "w")       # the order of the mixes, and of the products that read them

    def __init__(self, hidden: int, heads: int, dim: int, eps: float = 1e-6, decay_rank: int | None = None):
        self.hidden, self.heads, self.dim, self.eps, self.decay_rank = hidden, heads, dim, float(eps), decay_rank
        self.chunk = 128
        self.mu = self.w_in = self.w_w2 = self.b_w0 = self.u = self.w_norm = self.w_o = None

    def params(self):
        W, C, r = self.hidden, self.heads * self.dim, -1 if self.decay_rank is None else self.decay_rank
        return [Param("mu", tuple(Source("mu." + s, (W,)) for s in self.SHIFTED), role="vector"),
                Param("w_in", tuple(Source(s, (C, W)) for s in self.SHIFTED[:4]) + (Source("w1", (r, W)),)),
                Param("w_w2", (Source("w2", (C, r)),)),
                Param("b_w0", (Source("w0", (C,)),), role="vector"),
                Param("u", (Source("u", (self.heads, self.dim)),), role="vector"),
                Param("w_norm", (Source("norm", (C,), init="norm"),), role="vector"),
                Param("w_o", (Source("o", (W, C)),))]

    def cache_spec(self):
        return StateSpec((("S", (self.heads, self.dim, self.dim), torch.float32), ("prev", (self.hidden,), torch.float32)))

    def finalize(self, device, dtype):
        C = self.heads * self.dim
        f32 = lambda t: t.float().contiguous()
        self._mu, self._w0, self._u, self._norm_f32 = f32(self.mu).view(5, self.hidden), f32(self.b_w0), f32(self.u), f32(self.w_norm)
        self._rank = self.w_in.shape[0] - 4 * C
        self._w2_t = self.w_w2.t().contiguous()          # the kernel's lanes own columns
        if self.w_w2.shape[1] != self._rank:
            raise ValueError(f"{self.prefix}w1 has {self._rank} rows, w2 takes {self.w_w2.shape[1]}")

    def forward_stream(self, h, norm, ctx, cache, second=None):
        """h: the float stream. Returns the float output and the rows of the `second` norm (weight, eps) of h, or None."""
        be = ctx.backend
        H, d, C = self.heads, self.dim, self.heads * self.dim
        x, n2 = be.shift_mix(h, norm.weight_f32(), norm.eps, self._mu, ctx, cache.state["prev"], second)    # [T, 5, W]
        proj = be.linear_mixes(x, self.w_in, C, tag="in")                # [T, r | k | v | g | w1]
        decay = be.lowrank_decay(proj[:, 4 * C:], self._w2_t, self._w0)   # float [T, C]
        o = be.gla_scan(proj, 0, C, 2 * C, decay, 1.0, H, d, d, ctx.cu_q, ctx.num_seqs, ctx.state_slots, cache.state["S"],
                        scan_chunk(ctx, self.chunk), bonus=self._u)
        return be.linear_f32(be.gla_finish(o, self._norm_f32, self.eps, proj, 3 * C), self.w_o, tag="o"), n2


register_part("mixer", "gla", GatedLinearAttention)
register_part("mixer", "time_mixing", TimeMixing)
