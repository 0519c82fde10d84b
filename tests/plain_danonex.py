"""A plain, slow Danonex on the CPU: the tests' yardstick for the package's Danonex parts.

One function per mechanism, written from the design's equations with float64 torch tensors on the CPU and a python loop
over tokens where the design is recurrent. It shares no code with `rllm_b200`: its only inputs are the raw
`config.json` dictionary and the checkpoint's tensors by name.

Notation: x is the residual stream [T, width], which the sublayers read as it is; positions count from 0; `eps` is
`norm.eps`; a weight W is stored [out, in] and applied as x @ W.T; `p` is a mixer's tensor prefix. `stored` is what a
run does to the activations it keeps between two kernels (nothing, or a rounding).
"""
from __future__ import annotations

import math

import torch

from plain_purozen import read_model_dir, read_safetensors  # noqa: F401  (plain file readers, no model code)

DT = torch.float64


def exact(x):
    return x


# ------------------------------------------------------------------ small pieces

def rms_norm(x, w, eps):
    """w * x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    """log(1 + e^z), written so that neither end overflows."""
    return z.clamp(min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu_erf(z):
    """z times the standard normal distribution function."""
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


# ------------------------------------------------------------------ the gated delta rule

def causal_conv(y, kernel):
    """out[t, c] = silu(sum_j kernel[c, j] y[t - (taps - 1) + j, c]), inputs before the first token zero."""
    T, taps = y.shape[0], kernel.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, y.shape[1], dtype=y.dtype), y])
    return silu(sum(kernel[:, j] * padded[j: j + T] for j in range(taps)))


def unit_vectors(v):
    return v / torch.sqrt((v ** 2).sum(-1, keepdim=True) + 1e-6)


def head_decay(x, w, p):
    """One decay per token and head, between 0 and 1."""
    return torch.exp(-torch.exp(w[p + "A_log"]) * softplus(x @ w[p + "a"].T + w[p + "dt_bias"]))


def delta_steps(q, k, v, g, beta):
    """q, k [T, H, d], v [T, H, dv], g, beta [T, H]: per head, token by token, with S [d, dv] from zero,
    S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=DT)
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def delta_mixer(x, w, p, m, eps, stored=exact):
    T, H, G, d, dv = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = {n: causal_conv(stored(x @ w[p + n].T), w[p + n + ".conv"]) for n in "qkv"}
    q = unit_vectors(conv["q"].view(T, G, d)) * d ** -0.5
    k = unit_vectors(conv["k"].view(T, G, d))
    which = torch.arange(H) // (H // G)                     # the query/key head of each head
    o = delta_steps(q[:, which], k[:, which], conv["v"].view(T, H, dv), head_decay(x, w, p), torch.sigmoid(x @ w[p + "b"].T))
    o = rms_norm(o, w[p + "norm"], eps) * silu(stored(x @ w[p + "g"].T)).view(T, H, dv)
    return stored(o.reshape(T, H * dv)) @ w[p + "o"].T


# ------------------------------------------------------------------ attention

def yarn(f, rot):
    """The rotation's frequencies and the factor on its cosines and sines. Slow frequencies are divided by `factor`, fast
    ones kept, with a linear ramp over the index between the two indices where a frequency makes `fast` and `slow` turns
    over the original context."""
    s = rot.get("scaling")
    if s is None:
        return f, 1.0
    dims = rot["dims"]

    def index(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(rot["base"]))
    lo, hi = max(math.floor(index(s["fast"])), 0), min(math.ceil(index(s["slow"])), dims - 1)
    ramp = torch.clamp((torch.arange(len(f), dtype=DT) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate_interleaved(x, rot, positions):
    """x [T, heads, d]: of the first rot.dims numbers of a head, 2i and 2i + 1 turn together by position * f_i."""
    if rot is None or rot["dims"] == 0:
        return x
    n = rot["dims"] // 2
    f, mag = yarn(torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(n)], dtype=DT), rot)
    ang = positions.to(DT)[:, None, None] * f
    z = torch.view_as_complex(x[..., : 2 * n].reshape(*x.shape[:-1], n, 2).contiguous())
    z = z * torch.polar(torch.full_like(ang, mag), ang)
    return torch.cat([torch.view_as_real(z).flatten(-2), x[..., 2 * n:]], -1)


def capped(s, cap):
    return s if cap is None else cap * torch.tanh(s / cap)


def sink_softmax(s, seen, sink):
    """s [H, queries, keys]: weights over the seen keys whose denominator also holds exp(sink_h)."""
    s = s.masked_fill(~seen, float("-inf"))
    z = torch.cat([s, sink[:, None, None].expand(s.shape[0], s.shape[1], 1)], -1)
    return torch.softmax(z, -1)[..., :-1]


def attention(x, w, p, m, eps, stored=exact):
    T, H, G, d, dv = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(stored(x @ w[p + "q"].T), w[p + "q.norm"], eps)          # one norm over all heads together
    k = rms_norm(stored(x @ w[p + "k"].T), w[p + "k.norm"], eps)
    v = stored(x @ w[p + "v"].T).view(T, G, dv)
    pos = torch.arange(T)
    q = stored(rotate_interleaved(q.view(T, H, d), m.get("rot"), pos))
    k = stored(rotate_interleaved(k.view(T, G, d), m.get("rot"), pos))
    which = torch.arange(H) // (H // G)
    s = capped(torch.einsum("ihd,jhd->hij", q, k[:, which]) * m["scale"], m.get("softcap"))
    a = sink_softmax(s, pos[None, :] <= pos[:, None], w[p + "sink"])
    o = torch.einsum("hij,jhv->ihv", a, v[:, which]).reshape(T, H * dv)
    return stored(o) @ w[p + "o"].T


# ------------------------------------------------------------------ feed-forward, model

def feed_forward(x, w, p, stored=exact):
    return stored(gelu_erf(x @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, w, ids, keep_layers=False):
    """Logits [T, vocab] of one sequence (and the stream after every layer with `keep_layers`)."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.tensor(ids)]
    kept = []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = {"delta": delta_mixer, "attention": attention}[L["type"]]
        x = x + m * rms_norm(mixer(x, w, p + "mix.", L["mixer"], eps), w[p + "norm1"], eps)
        if L["mlp"] is not None:
            x = x + m * rms_norm(feed_forward(x, w, p + "mlp."), w[p + "norm2"], eps)
        kept.append(x.clone())
    logits = rms_norm(x, w["final.norm"], eps) @ w["embed"].T * cfg["logit_scale"]
    return (logits, kept) if keep_layers else logits


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
