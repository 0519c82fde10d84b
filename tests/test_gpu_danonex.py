"""Danonex on the GPU against the plain implementation (tests/plain_danonex.py): each mechanism alone, then whole models
through the step function, the scheduler, the command line and the trace program; prompts whole, in portions down to two
tokens, decoded token by token, and in mixed batches with pages and slots used again. Queries and keys are normed over
a whole row, so a larger input changes nothing; where random inputs would hide a fault, tokens are pointed the way of the
queries that should find them (a far key, keys at page borders, the first tokens), decays are made slow (the first
token is still felt at the end), and bounds and sinks are sized so that leaving one out moves the rows."""
import itertools
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import danonex_tiny as Z
import plain_danonex as P
import replay
from test_gpu_purozen import as_stored, bind, over_schedules, stored_as
from test_gpu_zukotar import SCHEDULES, Harness, check, cut, rel, rnd

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def built_mixer(W, layer, eps=1e-5):
    """The mixer part of a one-layer model, as the model builder makes it."""
    from rllm_b200.config import config_from_dict
    arch, cfg = config_from_dict(Z.model(10, W, eps, 1.0, 1.0, [layer]))
    return arch.build(cfg).blocks[0].mixer


# ------------------------------------------------------------------ small kernels

@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("H", [40, 96, 102, 1024, 5000])
def test_normed_output_into_the_stream(H, dtype):
    """h += m w y / rms(y): one summand, several parts, a gated second summand; the copy in the run's type."""
    from rllm_b200.kernels import sink
    T, m = 9, 0.37
    h, y, w = rnd(T, H, seed=1), rnd(T, 3, H, seed=2, scale=3.0), rnd(H, seed=3) + 1
    y2, zg = rnd(T, H, seed=4), rnd(T, 2, seed=5)
    for parts, second in ((1, False), (3, False), (3, True)):
        s = y[:, :parts].double().sum(1)
        if second:
            s = s + torch.sigmoid(zg[:, :1].double()) * y2.double()
        want = h.double() + m * P.rms_norm(s, w.double(), 1e-5)
        hd = h.to(DEV)
        copy = torch.empty(T, H, dtype=DT[dtype], device=DEV)
        yd = (y[:, 0] if parts == 1 else y[:, :parts]).contiguous().to(DEV)
        sink.postnorm(hd, yd, m, w.to(DEV), 1e-5, y2.to(DEV) if second else None, zg.to(DEV) if second else None, copy, output=True)
        assert rel(hd, want) < 2e-6 and torch.equal(copy, hd.to(DT[dtype]))
        # norming the sum instead is another thing
        assert rel(P.rms_norm(h.double() + m * s, w.double(), 1e-5), want) > 0.1
    hd = h.to(DEV)
    sink.postnorm(hd, torch.zeros(T, H, device=DEV), m, w.to(DEV), 1e-5, output=True)
    assert torch.equal(hd.cpu(), h)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("T,K,N", [(3, 64, 96), (40, 128, 320), (300, 256, 512), (2100, 128, 256), (5, 72, 100), (7, 50, 33)])
def test_erf_gelu_behind_a_product(dtype, T, K, N):
    """act(x W^T) as the feed-forward asks for it, with the activation on the float product, rounded once; inputs that
    reach both tails; with and without a norm in front."""
    from rllm_b200.kernels.backend import Backend
    be = Backend(DT[dtype], DEV)
    h, g, w = rnd(T, K, seed=1, scale=2.0), rnd(K, seed=2, scale=0.2) + 1, rnd(N, K, seed=3, scale=0.2)
    ws = w.to(DT[dtype]).double()
    x = (h * 0.5).to(DT[dtype])
    want = P.gelu_erf(x.double() @ ws.T)
    got = be.linear_act(x.to(DEV), w.to(DT[dtype]).to(DEV), "gelu_erf")
    assert got.dtype == DT[dtype] and rel(got, want) < (2e-6 if dtype == "float32" else 5e-3)
    tanh_form = 0.5 * (x.double() @ ws.T) * (1 + torch.tanh(0.7978845608028654 * ((x.double() @ ws.T) + 0.044715 * (x.double() @ ws.T) ** 3)))
    if dtype == "float32":
        assert rel(tanh_form, want) > 1e-5              # the two forms are told apart
    n = P.rms_norm(h.double(), g.double(), 1e-5)
    got = be.linear_act(be.normed(h.to(DEV), g.to(DEV), 1e-5), w.to(DT[dtype]).to(DEV), "gelu_erf")
    assert rel(got, P.gelu_erf(stored_as(dtype)(n) @ ws.T)) < (2e-5 if dtype == "float32" else 1.5e-2)


def half_split(x, rot, positions):
    """The other pairing (number i with i + dims/2), by reordering."""
    n = rot["dims"] // 2
    order = torch.stack([torch.arange(n), torch.arange(n) + n], 1).flatten()
    y = P.rotate_interleaved(torch.cat([x[..., order], x[..., 2 * n:]], -1), rot, positions)
    out = y.clone()
    out[..., order] = y[..., : 2 * n]
    return out


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("nh,nkv,kd,vd,dims", [
    (4, 2, 24, 40, 16), (3, 1, 20, 12, 6), (2, 2, 64, 64, 64), (32, 8, 128, 128, 64), (5, 5, 8, 16, 0), (70, 2, 64, 32, 20),
    (16, 4, 128, 64, 2), (1, 1, 6, 4, 4), (128, 128, 128, 128, 128)])
@pytest.mark.parametrize("span", ["row", "head"])
def test_query_key_norm_rotation_and_cache_write(dtype, nh, nkv, kd, vd, dims, span):
    """The norm over a token's whole row and over each head, both pairings of the rotation with scaled frequencies and the
    factor on cosines and sines, keys and values in their pages, tokens without a slot; what lies beside q, k, v in the
    rows stays. Rows longer than a thread block's registers take the staged kernel."""
    from rllm_b200.config.danonex import YarnScaling
    from rllm_b200.kernels import ops, sink
    from rllm_b200.parts import inverse_frequencies
    from rllm_b200.parts.rope import table_magnitude
    if nh * kd > 8192 and span == "head":
        pytest.skip("row lengths matter to the row norm only")
    T, page, eps = 11, 4, 1e-5
    rot = {"base": 700.0, "dims": dims, "scaling": {"factor": 3.0, "original": 50, "fast": 4.0, "slow": 0.5}}
    q_off, k_off = 8, 8 + nh * kd
    v_off = k_off + nkv * kd
    cols = v_off + nkv * vd + 8
    proj = rnd(T, cols, seed=nh).to(DT[dtype])
    proj[:, q_off: q_off + kd] *= 4.0                       # one head larger than the rest: the two spans differ
    proj[:, k_off: k_off + kd] *= 4.0
    nq, nk = (nh * kd, nkv * kd) if span == "row" else (kd, kd)
    wq, wk = rnd(nq, seed=2, scale=0.3) + 1, rnd(nk, seed=3, scale=0.3) + 1
    positions = torch.arange(T) * 37 + 5
    slots = torch.randperm(40)[:T].int()
    slots[4] = -1

    def normed(x, w, heads):
        if span == "row":
            return P.rms_norm(x, w, eps).view(T, heads, kd)
        return P.rms_norm(x.view(T, heads, kd), w, eps)
    x = proj.double()
    q, k = normed(x[:, q_off:k_off], wq.double(), nh), normed(x[:, k_off:v_off], wk.double(), nkv)
    tol = 1.5e-5 if dtype == "float32" else 6e-3           # angles of several hundred, in float
    sc = YarnScaling(3.0, 50.0, 4.0, 0.5)
    table = None
    if dims:
        f = torch.tensor(inverse_frequencies(dims, 700.0, sc)).float()
        table = ops.rope_table(positions.int().to(DEV), f.to(DEV), T, table_magnitude(dims, 700.0, sc))
    for interleaved in ((True, False) if dims else (True,)):
        turn = (lambda z: z) if not dims else (lambda z: (P.rotate_interleaved if interleaved else half_split)(z, rot, positions))
        kc = torch.zeros(10, nkv, page, kd, dtype=DT[dtype], device=DEV)
        vc = torch.zeros(10, nkv, page, vd, dtype=DT[dtype], device=DEV)
        pd = proj.to(DEV)
        sink.qk_norm_rope_store(pd, q_off, k_off, v_off, nh, nkv, kd, vd, dims, wq.to(DEV), wk.to(DEV), eps, table, slots.to(DEV), kc,
                                vc, row_norm=span == "row", interleaved=interleaved)
        assert rel(pd[:, q_off:k_off], turn(q).reshape(T, -1)) < tol
        keep = torch.ones(cols, dtype=torch.bool)
        keep[q_off:k_off] = False
        assert torch.equal(pd.cpu()[:, keep], proj[:, keep])
        kt = turn(k)
        for t in range(T):
            s = int(slots[t])
            if s < 0:
                continue
            assert rel(kc[s // page, :, s % page], kt[t]) < tol
            assert torch.equal(vc[s // page, :, s % page].cpu(), proj[t, v_off: v_off + nkv * vd].view(nkv, vd))
        assert int((vc.abs().sum((1, 3)) > 0).sum()) == T - 1
    # no norm; and a step that stores nothing
    pd = proj.to(DEV)
    sink.qk_norm_rope_store(pd, q_off, k_off, v_off, nh, nkv, kd, vd, dims, None, None, eps, table, None, None, None,
                            row_norm=span == "row", interleaved=True)
    assert rel(pd[:, q_off:k_off], (P.rotate_interleaved(x[:, q_off:k_off].view(T, nh, kd), rot, positions)).reshape(T, -1)) < tol


# ------------------------------------------------------------------ the delta rule, over steps and slots

def delta_weights(W, m, seed):
    H, G, d, v, c = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    shapes = {"q": (G * d, W), "q.conv": (G * d, c), "k": (G * d, W), "k.conv": (G * d, c), "v": (H * v, W), "v.conv": (H * v, c),
              "b": (H, W), "a": (H, W), "A_log": (H,), "dt_bias": (H,), "norm": (v,), "g": (H * v, W), "o": (W, H * v)}
    w = {"x." + k: rnd(*s, seed=seed + i, scale=0.3 if len(s) == 2 else 1.0) for i, (k, s) in enumerate(shapes.items())}
    for n in "qkv":
        w[f"x.{n}.conv"] = rnd(*shapes[n + ".conv"], seed=seed + 60, scale=0.8)
    w["x.A_log"] -= 4.0                  # slow decays: the first token is still felt at the end
    w["x.norm"] = w["x.norm"] * 0.3 + 1
    return w


DELTAS = [Z.delta(4, 2, 24, 16, 4, None), Z.delta(3, 1, 10, 14, 1, None), Z.delta(2, 2, 32, 64, 2, None), Z.delta(4, 4, 64, 40, 3, None),
          Z.delta(6, 3, 1, 6, 5, None), Z.delta(2, 1, 128, 128, 4, None), Z.delta(1, 1, 70, 9, 3, None), Z.delta(16, 8, 16, 8, 4, None),
          Z.delta(2, 1, 256, 24, 9, None)]


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("layer", DELTAS)
def test_delta_rule_over_steps_and_slots(dtype, layer):
    W, n, eps, m = 40, 97, 1e-5, layer["mixer"]
    w = delta_weights(W, m, seed=m["dim"])
    h = rnd(n, W, seed=9)
    h[0] *= 3.0
    x = h.to(DT[dtype])
    st, sa = as_stored(w, dtype), stored_as(dtype)
    want = P.delta_mixer(x.double(), st, "", m, eps, stored=sa)
    # felt: the first token at the end; the decay; the taps before the current one
    x0 = x.double().clone()
    x0[0] = 0
    if m["dim"] > 1:                     # (with one channel every write replaces most of what there was)
        assert rel(P.delta_mixer(x0, st, "", m, eps)[-1:], want[-1:]) > 1e-3
    assert rel(P.delta_mixer(x.double(), dict(st, A_log=st["A_log"] - 50), "", m, eps), want) > 1e-2
    part = built_mixer(W, layer, eps)
    bind(part, w, dtype, "x.")
    hd = x.to(DEV)
    tol = 3e-5 if dtype == "float32" else 3e-2

    def step(hs, entries, spans):
        rows = torch.cat([hd[a:b] for a, b in spans.values()])
        return hs.run(entries, lambda ctx, cache: part.forward(rows, ctx, cache))
    over_schedules(dtype, n, step, lambda: Harness(dtype, [part.cache_spec()], slots=2), want, tol)
    # two requests in one step, unequal portions beside single tokens; then a third in a slot that was used
    hb = rnd(47, W, seed=10).to(DT[dtype])
    want_b = P.delta_mixer(hb.double(), st, "", m, eps, stored=sa)
    hbd = hb.to(DEV)
    hs = Harness(dtype, [part.cache_spec()], slots=2)
    got_a, got_b, ia, ib = [], [], 0, 0
    for qa, qb in ((30, 5), (1, 40), (66, 2)):
        y = hs.run([("a", qa), ("b", qb)], lambda ctx, cache: part.forward(torch.cat([hd[ia: ia + qa], hbd[ib: ib + qb]]), ctx, cache))
        got_a.append(y[:qa]); got_b.append(y[qa:])
        ia += qa; ib += qb
    assert rel(torch.cat(got_a), want) < tol and rel(torch.cat(got_b), want_b) < tol
    hs.engine.end(["a", "b"])
    again = hs.run([("c", 47)], lambda ctx, cache: part.forward(hbd, ctx, cache))       # starts from zero
    assert rel(again, want_b) < tol


# ------------------------------------------------------------------ attention, over steps

def att_weights(W, m, seed):
    """Input channel 0 feeds one direction per key/value head into the keys and into the queries of the heads that read
    them: tokens with a large channel 0 find each other. The direction lies in the part of a head that turns slowly or
    not at all, so that distance does not undo it."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    shapes = {"q": (H * D, W), "k": (G * D, W), "v": (G * V, W), "o": (W, H * V)}
    w = {"x." + k: rnd(*s, seed=seed + i, scale=0.25) for i, (k, s) in enumerate(shapes.items())}
    a = rnd(G, D, seed=seed + 50)
    dims = (m.get("rot") or {"dims": 0})["dims"]
    if dims < D:
        a[:, :dims] = 0.0
    else:
        a[:, : D - 4] = 0.0
    w["x.k"][:, 0] = a.reshape(-1)
    w["x.q"][:, 0] = a.repeat_interleave(H // G, 0).reshape(-1)
    w["x.q.norm"], w["x.k.norm"] = rnd(H * D, seed=seed + 8, scale=0.3) + 1, rnd(G * D, seed=seed + 9, scale=0.3) + 1
    w["x.sink"] = rnd(H, seed=seed + 10) + 2.0
    return w


ATTS = [
    (Z.att(4, 2, 24, 40, 0.3, None, 6.0, (800.0, 16, (4.0, 64, 8.0, 1.0))), 4),        # heads that share keys, several pages
    (Z.att(3, 3, 16, 24, 0.4, None, 20.0, (1e5, 16, (2.5, 100, 3.0, 0.5))), 16),       # as many key/value heads; the whole head turns
    (Z.att(5, 1, 12, 12, 0.5, None), 8),                                               # no bound, no rotation
    (Z.att(6, 3, 20, 10, 0.4, None, 2.5, (50.0, 8, None)), 16),                        # nothing a multiple of 8 but the rotation
    (Z.att(4, 2, 64, 64, 0.12, None, 5.0, (20000.0, 32, (8.0, 512, 16.0, 2.0))), 16),  # equal sizes of 64
    (Z.att(2, 1, 128, 128, 0.08, None, 7.0, (1e7, 128, (3.0, 2048, 64.0, 1.0))), 16),  # equal sizes of 128
    (Z.att(16, 2, 32, 48, 0.25, None, 5.0, (300.0, 20, (2.0, 40, 2.0, 1.0))), 16),     # many heads a key
    (Z.att(2, 2, 80, 16, 0.1, None, 50.0, (5000.0, 40, (1.0, 128, 4.0, 4.0))), 8),     # a bound that hardly bites
    (Z.att(1, 1, 200, 136, 0.05, None, 4.0, (100.0, 6, (5.0, 30, 1.5, 1.0))), 4),      # heads beyond the tensor-core kernels
]


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("layer,page", ATTS)
def test_attention_over_steps(dtype, layer, page):
    W, n, eps, m = 40, 97, 1e-5, layer["mixer"]
    w = att_weights(W, m, seed=m["heads"])
    h = rnd(n, W, seed=9)
    marked = sorted({0, 1, page - 1, page, 2 * page + 1, 50, 70, 96})
    for p in marked:
        h[p, 0] += 12.0
    x = h.to(DT[dtype])
    st, sa = as_stored(w, dtype), stored_as(dtype)
    want = P.attention(x.double(), st, "", m, eps, stored=sa)
    # the yardstick itself moves with what is tested: the bound, the sink, the scaling, the far keys
    moved = lambda y: rel(y, want)
    if m.get("softcap", 99) < 20:
        assert moved(P.attention(x.double(), st, "", {k: v for k, v in m.items() if k != "softcap"}, eps)) > 1e-2
    assert moved(P.attention(x.double(), dict(st, sink=st["sink"] - 50), "", m, eps)) > 1e-2
    for p in marked[:-1]:
        x0 = x.double().clone()
        x0[p] = x0[p] * 0.5 - x0[(p + 5) % n]
        assert rel(P.attention(x0, st, "", m, eps)[-1:], want[-1:]) > 1e-2, p
    if m.get("rot", {}).get("scaling", {}).get("factor", 1.0) != 1.0:
        off = dict(m, rot={k: v for k, v in m["rot"].items() if k != "scaling"})
        assert moved(P.attention(x.double(), st, "", off, eps)) > 1e-2
    part = built_mixer(W, layer, eps)
    bind(part, w, dtype, "x.")
    hd = x.to(DEV)
    tol = 3e-5 if dtype == "float32" else 3e-2

    def step(hs, entries, spans):
        rows = torch.cat([hd[a:b] for a, b in spans.values()])
        return hs.run(entries, lambda ctx, cache: part.forward(rows, ctx, cache))
    over_schedules(dtype, n, step, lambda: Harness(dtype, [part.cache_spec()], page_size=page, pages=2 + (n + page - 1) // page),
                   want, tol)
    # two requests in one step, unequal portions beside single tokens; then a third on pages that were used
    hb = rnd(47, W, seed=10)
    hb[3, 0] += 12.0
    hb[40, 0] += 12.0
    xb = hb.to(DT[dtype])
    want_b = P.attention(xb.double(), st, "", m, eps, stored=sa)
    hbd = xb.to(DEV)
    hs = Harness(dtype, [part.cache_spec()], page_size=page, pages=4 + (n + 47 + 2 * page - 1) // page)
    got_a, got_b, ia, ib = [], [], 0, 0
    for qa, qb in ((30, 5), (1, 40), (66, 2)):
        y = hs.run([("a", qa), ("b", qb)], lambda ctx, cache: part.forward(torch.cat([hd[ia: ia + qa], hbd[ib: ib + qb]]), ctx, cache))
        got_a.append(y[:qa]); got_b.append(y[qa:])
        ia += qa; ib += qb
        hs.cache.check()
    assert rel(torch.cat(got_a), want) < tol and rel(torch.cat(got_b), want_b) < tol
    hs.engine.end(["a", "b"])
    again = hs.run([("c", 47)], lambda ctx, cache: part.forward(hbd, ctx, cache))
    assert rel(again, want_b) < tol


def paged(lens, nkv, kd, vd, page, n_pages, g, dtype, spread=1.0):
    """Random keys and values of several sequences in scattered pages: (k, v by sequence, pages, table)."""
    k = [(torch.randn(n, nkv, kd, generator=g) * spread).to(dtype) for n in lens]
    v = [torch.randn(n, nkv, vd, generator=g).to(dtype) for n in lens]
    S = len(lens)
    kc = torch.zeros(n_pages * S, nkv, page, kd, dtype=dtype)
    vc = torch.zeros(n_pages * S, nkv, page, vd, dtype=dtype)
    bt = torch.randperm(n_pages * S, generator=g).int().view(S, n_pages).contiguous()

    def store():
        for s in range(S):
            j = torch.arange(lens[s])
            kc[bt[s][j // page].long(), :, j % page], vc[bt[s][j // page].long(), :, j % page] = k[s], v[s]
        return kc.to(DEV), vc.to(DEV), bt.to(DEV)
    return k, v, store


def plain_bounded(q, k, v, lens, qlens, nh, nkv, scale, cap, sinks):
    """q rows of every sequence's last positions over its keys -> [T, nh * vd] in float64."""
    out, r = [], 0
    for s, n in enumerate(lens):
        kk, vv = (t.double().repeat_interleave(nh // nkv, 1) for t in (k[s], v[s]))
        for i in range(n - qlens[s], n):
            sc = P.capped(torch.einsum("hd,jhd->hj", q[r].double(), kk[: i + 1]) * scale, cap)
            p = P.sink_softmax(sc[:, None], torch.ones(1, i + 1, dtype=torch.bool), sinks.double())[:, 0]
            out.append(torch.einsum("hj,jhv->hv", p, vv[: i + 1]).reshape(-1))
            r += 1
    return torch.stack(out)


@pytest.mark.parametrize("cap", [2.0, 15.0, 60.0, None])
@pytest.mark.parametrize("kd,vd", [(64, 48), (48, 80), (128, 128)])
def test_bounded_scores_in_long_contexts_on_cuda_cores_and_mma(cap, kd, vd):
    """Contexts of up to 1,100 keys over scattered pages, single tokens and a portion in one launch; one far key scores
    beyond every bound for the marked query, so that it wins the unbounded softmax and only shares a small bound's. The
    tensor-core kernel also with the keys of a row tile dealt out to several CTAs, and in its form for single tokens."""
    from rllm_b200.kernels import sink
    g = torch.Generator().manual_seed(kd)
    nh, nkv, page, n_pages, scale = 8, 2, 16, 70, 1.0 / kd ** 0.5
    lens, qlens = [900, 333, 1100, 1], [1, 1, 40, 1]
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        k, v, store = paged(lens, nkv, kd, vd, page, n_pages, g, dtype)
        q = torch.cat([torch.randn(ql, nh, kd, generator=g) for ql in qlens]).to(dtype)
        for far in (0, 15, 16, 99):
            k[0][far] = q[0][::4] * 4
        sinks = torch.randn(nh, generator=g) + 1
        want = plain_bounded(q, k, v, lens, qlens, nh, nkv, scale, cap, sinks)
        if cap is not None and cap < 10:
            assert rel(plain_bounded(q[:1], k, v, lens[:1], [1], nh, nkv, scale, None, sinks), want[:1]) > 1e-2
        kc, vc, bt = store()
        pos = torch.cat([torch.arange(n - ql, n) for n, ql in zip(lens, qlens)]).int().to(DEV)
        seq = torch.cat([torch.full((ql,), i) for i, ql in enumerate(qlens)]).int().to(DEV)
        qd, sd = q.reshape(-1, nh * kd).to(DEV), sinks.to(DEV)
        got = sink.sink_attention_simt(qd, kc, vc, seq, pos, bt, nh, scale, None, None, sd, softcap=cap)
        assert rel(got, want) < tol, dtype
        if dtype == torch.bfloat16:
            assert sink.mma_supported(dtype, kd, vd, page)
            cu = torch.tensor([0] + list(itertools.accumulate(qlens)), dtype=torch.int32, device=DEV)
            for splits in (1, 3):
                got = sink.sink_attention_mma(qd, kc, vc, seq, pos, bt, cu, 4, 40, nh, scale, None, None, sd, None, splits, 1100, softcap=cap)
                assert rel(got, want) < tol, splits
            one = [0, 1, 42]
            cu1 = torch.arange(4, dtype=torch.int32, device=DEV)
            for splits in (1, 4):
                got = sink.sink_attention_mma(qd[one], kc, vc, seq[one], pos[one], bt[[0, 1, 3]].contiguous(), cu1, 3, 1, nh, scale, None, None,
                                              sd, None, splits, 1100, softcap=cap)
                assert rel(got, want[one]) < tol, splits


@pytest.mark.parametrize("hd", [64, 128])
@pytest.mark.parametrize("cap", [1.5, 15.0, 60.0])
@pytest.mark.parametrize("G", [1, 4, 16])
def test_bounded_scores_on_the_decode_and_the_tcgen05_kernel(hd, cap, G):
    """Equal head sizes of 64 or 128. The tcgen05 kernel bounds scores by a polynomial where all of a warp's rows lie
    within the bound and by the exponential form where one lies beyond; both are run (with a bound of 60 nothing but the
    marked keys comes near). Portions with all keys in the step, behind cached keys, and short; keys ranges merged in a
    cluster for single tokens."""
    from rllm_b200.kernels import sink, sm100
    g = torch.Generator().manual_seed(hd + G)
    nkv = 2
    nh, page, n_pages, scale = nkv * G, 16, 45, 1.0 / hd ** 0.5
    lens, qlens = [700, 420, 300], [300, 420, 130]
    k, v, store = paged(lens, nkv, hd, hd, page, n_pages, g, torch.bfloat16)
    q = torch.cat([torch.randn(ql, nh, hd, generator=g) for ql in qlens]).bfloat16()
    for far in (0, 15, 16, 399, 640):
        k[0][far] = q[299][:: G] * 3
    sinks = torch.randn(nh, generator=g) + 1
    kc, vc, bt = store()
    T = sum(qlens)
    pos = torch.cat([torch.arange(n - ql, n) for n, ql in zip(lens, qlens)]).int().to(DEV)
    seq = torch.cat([torch.full((ql,), i) for i, ql in enumerate(qlens)]).int().to(DEV)
    cu = torch.tensor([0, 300, 720, 850], dtype=torch.int32, device=DEV)
    kv = torch.tensor(lens, dtype=torch.int32, device=DEV)
    qd, sd = q.reshape(T, nh * hd).to(DEV), sinks.to(DEV)
    # the float kernel against plain arithmetic on a few rows, then everything against the float kernel
    want = sink.sink_attention_simt(qd, kc, vc, seq, pos, bt, nh, scale, None, None, sd, softcap=cap)
    last = [299, 719, 849]
    plain = plain_bounded(q[last], k, v, lens, [1, 1, 1], nh, nkv, scale, cap, sinks)
    assert rel(want[last], plain) < 1e-2
    unbounded = sink.sink_attention_simt(qd, kc, vc, seq, pos, bt, nh, scale, None, None, sd)
    assert cap > 20 or rel(unbounded, want) > 2e-2
    got = sm100.attention_prefill_tc(qd, kc, vc, cu, kv, bt, max(qlens), nh, scale, None, sinks=sd, softcap=cap)
    sm100.check_error(DEV)
    assert rel(got, want) < 2e-2
    for splits in (1, 3, 8):
        got = sm100.attention_decode(qd[last].contiguous(), kc, vc, kv, bt, nh, scale, None, 700, splits=splits, sinks=sd, softcap=cap)
        assert rel(got, plain) < 2e-2, splits


def test_the_engine_sends_long_portions_and_single_tokens_to_the_fast_kernels():
    """Heads of 64 / 64: a portion of 700 tokens behind 200 cached ones runs on the tcgen05 kernel, single tokens on the
    cluster kernel; both with the bound and the sink, against the plain implementation."""
    from rllm_b200.kernels import sm100
    W, n, eps, dtype = 64, 940, 1e-5, "bfloat16"
    layer = Z.att(4, 2, 64, 64, 0.12, None, 5.0, (20000.0, 32, (8.0, 512, 16.0, 2.0)))
    w = att_weights(W, layer["mixer"], 3)
    h = rnd(n, W, seed=9)
    for p in (0, 15, 16, 199, 200, 500, 899, 939):
        h[p, 0] += 12.0
    x = h.to(DT[dtype])
    want = P.attention(x.double(), as_stored(w, dtype), "", layer["mixer"], eps, stored=stored_as(dtype))
    part = built_mixer(W, layer, eps)
    bind(part, w, dtype, "x.")
    calls = {"tc": 0, "decode": 0}
    real_tc, real_dec = sm100.attention_prefill_tc, sm100.attention_decode
    sm100.attention_prefill_tc = lambda *a, **k: (calls.__setitem__("tc", calls["tc"] + 1), real_tc(*a, **k))[1]
    sm100.attention_decode = lambda *a, **k: (calls.__setitem__("decode", calls["decode"] + 1), real_dec(*a, **k))[1]
    try:
        hs = Harness(dtype, [part.cache_spec()], page_size=16, pages=64)
        hd = x.to(DEV)
        got, i = [], 0
        for qn in [200, 700] + [1] * 40:
            got.append(hs.run([("a", qn)], lambda ctx, cache: part.forward(hd[i: i + qn], ctx, cache)))
            i += qn
        sm100.check_error(DEV)
    finally:
        sm100.attention_prefill_tc, sm100.attention_decode = real_tc, real_dec
    assert calls == {"tc": 1, "decode": 40}
    assert rel(torch.cat(got), want) < 3e-2


# ------------------------------------------------------------------ whole models

def requests_for(name, lens=(9, 61, 23, 150, 37, 2)):
    vocab = Z.TINY[name][0]["vocab"]
    return {f"r{i}": Z.random_prompt(n, vocab, 100 * len(name) + ord(name[1]) + i) for i, n in enumerate(lens)}


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("danonex")
    return {n: Z.make_model_dir(root, n) for n in Z.TINY}


@pytest.fixture(scope="module")
def plain(dirs):
    out = {}
    for name, d in dirs.items():
        cfg, w = P.read_model_dir(d)
        out[name] = {}
        for rid, toks in requests_for(name).items():
            lg = P.forward(cfg, w, toks).numpy()
            out[name].update({(rid, i): lg[i] for i in range(len(toks))})
    return out


FAMILIES = {"whole": replay.whole, "decode": lambda r: replay.prefill_then_decode(r, tail=40), "portions": replay.portions,
            "mixed": lambda r: replay.mixed(r, max_live=3)}


def engine_for(dirs, name, dtype, steps, reqs, max_requests=3):
    from rllm_b200.engine import load_engine
    return load_engine(dirs[name], dtype=dtype, page_size=Z.TINY[name][3],
                       max_tokens=replay.max_live_tokens(steps, reqs), max_requests=max_requests)


@pytest.mark.parametrize("name", list(Z.TINY))
def test_residual_stream_after_every_layer(dirs, name):
    """In float32, layer by layer: the first layer that differs names the mechanism."""
    from rllm_b200.engine import Entry, load_engine
    cfg, w = P.read_model_dir(dirs[name])
    toks = Z.random_prompt(45, cfg["vocab"], 9)
    _, kept = P.forward(cfg, w, toks, keep_layers=True)
    eng = load_engine(dirs[name], dtype="float32", page_size=Z.TINY[name][3], max_tokens=64, max_requests=1)
    got = []
    for b in eng.model.blocks:          # a block adds to the stream it is given, in place

        def wrap(h, ctx, cache, f=b.forward):
            out = f(h, ctx, cache)
            got.append(h.detach().float().cpu().clone())
            return out
        b.forward = wrap
    eng.step([Entry("a", toks, [])])
    assert len(got) == len(kept)
    for i, (g, k) in enumerate(zip(got, kept)):
        assert rel(g, k) < 3e-5, f"{name}: the stream differs after layer {i} ({cfg['layers'][i]['type']})"


@pytest.mark.parametrize("family", list(FAMILIES))
@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("name", list(Z.TINY))
def test_family_matches_plain(dirs, plain, name, dtype, family):
    """The pool holds just what the live requests need and there are three state slots for six requests: pages and
    slots are used again."""
    reqs = requests_for(name)
    steps = FAMILIES[family](reqs)
    eng = engine_for(dirs, name, dtype, steps, reqs)
    got = replay.run_in_process(eng, steps)
    eng.check()
    if dtype == "float32":
        check(got, plain[name], 5e-5, f"{name} float32 {family}")
    else:
        check(got, plain[name], 6e-2, f"{name} bfloat16 {family}", allow=0.02)


@pytest.mark.parametrize("name", list(Z.TINY))
def test_float32_is_the_same_however_it_is_cut(dirs, name):
    reqs = requests_for(name)
    ref = None
    for family, make in FAMILIES.items():
        steps = make(reqs)
        got = replay.run_in_process(engine_for(dirs, name, "float32", steps, reqs), steps)
        if ref is None:
            ref = got
        else:
            worst = max(float(np.abs(got[k] - ref[k]).max()) / float(np.abs(ref[k]).max()) for k in ref)
            assert worst <= 1e-5, f"{name} {family}: differs from whole prompts by {worst}"


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-5), ("bfloat16", 6e-2)])
def test_long_decoding_through_graphs(dirs, dtype, tol):
    """Two requests decoded side by side for 120 steps from prompts of 3 and 30 tokens: states and convolution tails are
    carried through replayed graphs, keys of decoded tokens fill page after page."""
    from rllm_b200.engine import Entry, load_engine
    name = "DA"
    cfg, w = P.read_model_dir(dirs[name])
    toks = {"x": Z.random_prompt(123, cfg["vocab"], 5), "y": Z.random_prompt(150, cfg["vocab"], 6)}
    want = {k: P.forward(cfg, w, t).numpy() for k, t in toks.items()}
    eng = load_engine(dirs[name], dtype=dtype, page_size=4, max_tokens=320, max_requests=2)
    eng.step([Entry("x", toks["x"][:3], []), Entry("y", toks["y"][:30], [])])
    got = {}
    for i in range(120):
        lg = eng.step([Entry("x", [toks["x"][3 + i]], [0]), Entry("y", [toks["y"][30 + i]], [0])]).float().cpu().numpy()
        got[("x", 3 + i)], got[("y", 30 + i)] = lg[0], lg[1]
        eng.cache.check()
    eng.check()
    assert eng.graphs is not None and eng.graph_steps == 120
    check(got, {(k, i): want[k][i] for (k, i) in got}, tol, f"long decoding {dtype}", allow=0.0 if dtype == "float32" else 0.02)


def test_long_prompts_in_portions_and_decoding_on_the_fast_kernels(dirs):
    """Heads of 64 and 128 (DD): prompts of 1,300 and 700 tokens in portions of 600, so that the tcgen05 kernel works
    inside the engine, then single tokens on the cluster kernel; on pages and slots that went back to the pool."""
    from rllm_b200.engine import Entry, load_engine
    cfg, w = P.read_model_dir(dirs["DD"])
    toks = {"x": Z.random_prompt(1320, cfg["vocab"], 5), "y": Z.random_prompt(720, cfg["vocab"], 6)}
    want = {k: P.forward(cfg, w, t).numpy() for k, t in toks.items()}
    eng = load_engine(dirs["DD"], dtype="bfloat16", page_size=16, max_tokens=1344, max_requests=1)
    for rid in ("y", "x"):
        t, got, i, n = toks[rid], {}, 0, len(toks[rid])
        for q in [600] * ((n - 20) // 600) + [(n - 20) % 600] + [1] * 20:
            lg = eng.step([Entry(rid, t[i: i + q], [0, q - 1] if q > 1 else [0])]).float().cpu().numpy()
            got[(rid, i)] = lg[0]
            got[(rid, i + q - 1)] = lg[-1]
            i += q
        eng.end([rid])
        eng.check()
        check(got, {k: want[rid][k[1]] for k in got}, 6e-2, f"long prompt {rid}", allow=0.05)


@pytest.mark.parametrize("name", ["DB", "DC", "DF", "DG"])
def test_greedy_generation_through_the_entry_point(dirs, name):
    """LLM.generate (scheduler, sampler, run-ahead decoding) against greedy decoding with the plain model."""
    from rllm_b200.api import LLM
    from rllm_b200.sampling import SamplingParams
    cfg, w = P.read_model_dir(dirs[name])
    prompts = [Z.random_prompt(n, cfg["vocab"], 70 + n) for n in (4, 19, 33)]
    want = []
    for p in prompts:
        toks = list(p)
        for _ in range(12):
            lg = P.forward(cfg, w, toks)[-1]
            top2 = lg.topk(2).values
            toks.append(int(lg.argmax()))
            if float(top2[0] - top2[1]) < 1e-4 * float(lg.abs().max()):      # a close call: the rest of this prompt proves nothing
                break
        want.append(toks[len(p):])
    llm = LLM(dirs[name], dtype="float32", page_size=Z.TINY[name][3], num_pages=40, max_active=2, max_chunk=16)
    got = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12))
    for g, w_ in zip(got, want):
        assert g[: len(w_)] == w_
    llm.engine.cache.check()


def test_ten_requests_decode_in_a_padded_graph(dirs):
    """Ten requests decode side by side: their graph has more rows than requests; the stand-in rows have no state
    slot, pages or wanted logits, and must neither disturb the others nor touch a state."""
    from rllm_b200.engine import Entry, load_engine
    name = "DA"
    cfg, w = P.read_model_dir(dirs[name])
    toks = {i: Z.random_prompt(5 + 3 * i + 9, cfg["vocab"], 300 + i) for i in range(10)}
    want = {i: P.forward(cfg, w, t).numpy() for i, t in toks.items()}
    eng = load_engine(dirs[name], dtype="float32", page_size=4, max_tokens=10 * 64, max_requests=10)
    eng.step([Entry(i, t[:-9], []) for i, t in toks.items()])
    got = {}
    for k in range(9):
        lg = eng.step([Entry(i, [t[len(t) - 9 + k]], [0]) for i, t in toks.items()]).float().cpu().numpy()
        for row, (i, t) in enumerate(toks.items()):
            got[(i, len(t) - 9 + k)] = lg[row]
    eng.check()
    assert eng.graph_steps == 9
    check(got, {(i, p): want[i][p] for (i, p) in got}, 5e-5, "padded graph")


def test_command_line_runs_the_design(dirs):
    name = "DF"
    cfg, w = P.read_model_dir(dirs[name])
    prompt = Z.random_prompt(11, cfg["vocab"], 3)
    toks = prompt + P.greedy(cfg, w, prompt, 5)
    r = subprocess.run([sys.executable, os.path.join(replay.ROOT, "bin", "rllm"), "run", "--model", dirs[name],
                        "--prompt-ids", " ".join(map(str, prompt)), "--max-tokens", "5", "--temperature", "0",
                        "--dtype", "float32", "--kv-pages", "32"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.split()] == toks[len(prompt):]


@pytest.mark.parametrize("name,dtype", [("DA", "float32"), ("DE", "bfloat16")])
def test_trace_program_runs_the_design(dirs, plain, tmp_path, name, dtype):
    reqs = requests_for(name)
    steps = replay.mixed(reqs, max_live=4)
    got = replay.run_program(dirs[name], dtype, steps, str(tmp_path / "out"), replay.max_live_tokens(steps, reqs),
                             Z.TINY[name][0]["vocab"], extra_args=["--page-size", "16"])
    if dtype == "float32":
        check(got, plain[name], 5e-5, "trace program")
    else:
        check(got, plain[name], 6e-2, "trace program bfloat16", allow=0.02)
