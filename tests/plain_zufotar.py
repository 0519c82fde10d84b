"""A plain, slow Zufotar on the CPU: the tests' yardstick for the package's Zufotar parts.

One function per mechanism, written from the design's equations with float64 torch tensors on the CPU and python
loops over tokens where the design is a recurrence. It shares no code with `rllm_b200`: its only inputs are the raw
`config.json` dictionary and the checkpoint's tensors by name.

Notation: h is a sublayer's input [T, width]; positions count from 0; `eps` is `norm.eps`.
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch

DT = torch.float64


# ------------------------------------------------------------------ files

def read_safetensors(path):
    """name -> float64 tensor (integer tables stay integers)."""
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32, "F16": torch.float16, "F64": torch.float64}
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, ent in header.items():
        if name == "__metadata__":
            continue
        lo, hi = ent["data_offsets"]
        t = torch.frombuffer(bytearray(data[lo:hi]), dtype=kinds[ent["dtype"]]).reshape(ent["shape"])
        out[name] = t.to(DT) if t.is_floating_point() else t.clone()
    return out


def read_model_dir(d):
    with open(os.path.join(d, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(d, "model.safetensors"))


# ------------------------------------------------------------------ small pieces

def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last dimension (w None: no weight)."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def softcap(z, cap):
    return z if cap is None else cap * torch.tanh(z / cap)


# ------------------------------------------------------------------ rotation

def yarn(rot):
    """-> (the dims/2 frequencies of the rotation, the factor on cosines and sines)."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if s is None:
        return torch.tensor(f, dtype=DT), 1.0
    at = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), dims - 1)
    for i in range(dims // 2):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        f[i] = f[i] / s["factor"] * r + f[i] * (1 - r)
    return torch.tensor(f, dtype=DT), 0.1 * math.log(s["factor"]) + 1.0


def rotate_interleaved(x, rot, pos):
    """x [T, ..., D]: the first rot.dims of the last axis in pairs (2i, 2i+1); the rest pass unchanged."""
    f, mag = yarn(rot)
    dims = rot["dims"]
    a = pos.to(DT)[:, None] * f[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    cos, sin = (torch.cos(a) * mag).reshape(shape), (torch.sin(a) * mag).reshape(shape)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


# ------------------------------------------------------------------ mixers

def latent_attention(h, w, p, m, eps):
    """Attention over latents with a latent in front of the queries and an output gate as wide as the heads."""
    T = h.shape[0]
    H, dim, rot, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    cq = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).reshape(T, H, dim + rot)
    dkv = h @ w[p + "dkv"].T
    c = rms_norm(dkv[:, :rank], w[p + "dkv.norm"], eps)        # the latent: what a cache would keep
    q_plain, q_rot, k_rot = q[..., :dim], q[..., dim:], dkv[:, rank:]
    if rot:
        q_rot, k_rot = rotate_interleaved(q_rot, m["rot"], pos), rotate_interleaved(k_rot, m["rot"], pos)
    k_plain = (c @ w[p + "uk"].T).reshape(T, H, dim)
    v = (c @ w[p + "uv"].T).reshape(T, H, vdim)
    s = (torch.einsum("ihd,jhd->hij", q_plain, k_plain) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    s = s.masked_fill(~(pos[None, :] <= pos[:, None])[None], float("-inf"))
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v).reshape(T, H * vdim)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def token_shift(h, mu, before=None):
    """h + (h' - h) * mu with h' the row before (`before`, or zeros, for the first one)."""
    first = torch.zeros_like(h[:1]) if before is None else before[None]
    return h + (torch.cat([first, h[:-1]]) - h) * mu


def wkv_steps(r, k, v, decay, u, S=None):
    """r, k, decay [T, H, dim], v [T, H, vdim], u [H, dim] -> outputs [T, H, vdim] and the last state. What a
    token writes it reads times u; the decay takes effect on what later tokens read."""
    T, H, dim = r.shape
    S = torch.zeros(H, dim, v.shape[-1], dtype=DT) if S is None else S.clone()
    o = torch.zeros(T, H, v.shape[-1], dtype=DT)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return o, S


def wkv(h, w, p, m, eps):
    """Time mixing: token shift, decays from a two-step projection, the recurrence with a bonus, head norm, gate."""
    T, H, dim = h.shape[0], m["heads"], m["dim"]
    x = {s: token_shift(h, w[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((x[s] @ w[p + s].T).reshape(T, H, dim) for s in "rkv")
    decay = torch.exp(-torch.exp(torch.tanh(x["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).reshape(T, H, dim)
    o, _ = wkv_steps(r, k, v, decay, w[p + "u"])
    o = rms_norm(o, None, eps).reshape(T, H * dim) * w[p + "norm"]
    return (o * silu(x["g"] @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------ feed-forward

def dense(h, w, p, mlp):
    return gelu_erf(h @ w[p + "up"].T) @ w[p + "down"].T


def gated(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w_router, correction, r):
    """-> (chosen experts [T, top], their weights [T, top]) for router dictionary `r`."""
    s = torch.sigmoid(h @ w_router.T)
    c = s + correction
    T, E = s.shape
    g = r.get("groups")
    if g is not None:
        per = E // g["count"]
        best = c.reshape(T, g["count"], per).sort(-1, descending=True).values[..., :2].sum(-1)
        ok = torch.zeros(T, g["count"], dtype=torch.bool).scatter_(1, best.topk(g["keep"], dim=-1).indices, True)
        c = c.masked_fill(~ok[:, :, None].expand(T, g["count"], per).reshape(T, E), float("-inf"))
    idx = c.topk(r["top"], dim=-1).indices
    wt = s.gather(1, idx)
    return idx, wt / (wt.sum(-1, keepdim=True) + 1e-20) * r["scale"]


def moe(h, w, p, mlp):
    idx, wt = route(h, w[p + "router"], w[p + "correction"], mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(idx[t].tolist(), wt[t]):
            out[t] += s * gated(h[t], w, p + f"e{e}.")
    if mlp.get("shared") is not None:
        out = out + gated(h, w, p + "shared.") * torch.sigmoid(h @ w[p + "shared.sg"].T)
    return out


# ------------------------------------------------------------------ the model

MIXERS = {"latent_attention": latent_attention, "wkv": wkv}
FFS = {"dense": dense, "moe": moe}


def layer_runs(cfg):
    """[(layer index, pass number or None if the layer begins no pass)] in running order."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        for i in range(loop["start"], loop["stop"]):
            runs.append((i, t if i == loop["start"] else None))
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, w, ids, keep_layers=False):
    """Logits [T, vocab] of a whole sequence; with `keep_layers` also the residual stream after every layer run."""
    ids = torch.as_tensor(ids, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = x0 = w["embed"][ids] * cfg["embedding"]["scale"]
    seen = []
    for i, begins in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if begins is not None:
            if begins > 0:
                x = x + x0
            x = x + w["loop.step"][begins]
        y = MIXERS[L["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", L["mixer"], eps)
        if L.get("mlp") is not None:
            y = y + FFS[L["mlp"]["kind"]](rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", L["mlp"])
        x = x + y
        seen.append(x)
    logits = softcap(rms_norm(x, w["final.norm"], eps) @ w["embed"].T, cfg.get("logit_softcap"))
    return (logits, torch.stack(seen)) if keep_layers else logits


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
