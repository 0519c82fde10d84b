"""Zufotar on the GPU against the plain implementation (tests/plain_zufotar.py): each mechanism alone, then whole models
through the step function, the scheduler, the command line and the trace program; prompts whole, in portions down to two
tokens, decoded token by token, and in mixed batches with pages and slots used again. Where random inputs would hide a
fault they are made so that it shows: the input at a few positions is scaled up, so that its key wins every score it takes
part in (a far key, keys at page borders, the first tokens), decays are slow on half the channels (the first token is still
felt at the end), tokens of a portion's edge are large (the token before it is felt), router rows tell experts apart."""
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_zufotar as P
import replay
import zufotar_tiny as Z
from test_gpu_purozen import as_stored, bind, over_schedules
from test_gpu_zukotar import SCHEDULES, Harness, check, cut, rel, rnd

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def built_block(W, layer, eps=1e-5):
    """The block of a one-layer model, as the model builder makes it."""
    from rllm_b200.config import config_from_dict
    arch, cfg = config_from_dict(Z.model(10, W, 1.0, eps, None, None, [layer]))
    return arch.build(cfg).blocks[0]


# ------------------------------------------------------------------ small kernels

@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("mixes", [3, 5])
@pytest.mark.parametrize("W,lens", [(40, (5, 1, 7)), (37, (5, 1, 7)), (96, (700, 1, 402)), (102, (700, 1, 403)), (1024, (5, 1, 7)),
                                    (1300, (701, 1, 402)), (2048, (600, 1, 500)), (5000, (5, 1, 7)), (9000, (3, 1, 2))])
def test_norm_shift_and_mixes(dtype, W, lens, mixes):
    """Three sequences in one step, one of a single token: the row before a portion's first comes from its slot, a sequence
    without a slot begins with zeros; the slots afterwards hold each portion's last normed row, other slots stay."""
    from rllm_b200.kernels import mix
    eps, eps2 = 1e-5, 3e-4
    T = sum(lens)
    h, w, w2, mu = rnd(T, W, seed=1, scale=2.0), rnd(W, seed=2, scale=0.3) + 1, rnd(W, seed=3) + 1, torch.rand(mixes, W, generator=torch.Generator().manual_seed(8))
    prev = rnd(4, W, seed=4, scale=3.0)
    slots = [2, 0, -1]
    n = P.rms_norm(h.double(), w.double(), eps)
    want, i = [], 0
    after = prev.double().clone()
    for q, s in zip(lens, slots):
        before = prev[s].double() if s >= 0 else None
        want.append(torch.stack([P.token_shift(n[i: i + q], m.double(), before) for m in mu], 1))
        if s >= 0:
            after[s] = n[i + q - 1]
        i += q
    want = torch.cat(want)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    a, b = lens[0], lens[0] + 1
    seq, cu = i32([0] * a + [1] + [2] * lens[2]), i32([0, a, b, T])
    pd = prev.to(DEV)
    tol = 2e-6 if dtype == "float32" else 5e-3
    got, plain, second = mix.shift_mix(h.to(DEV), w.to(DEV), eps, DT[dtype], mu.to(DEV), seq, cu, 3, i32(slots), pd, plain=True,
                                       second=(w2.to(DEV), eps2))
    assert got.dtype == DT[dtype] and tuple(got.shape) == (T, mixes, W)
    assert rel(got, want) < tol and rel(plain, n) < tol and rel(second, P.rms_norm(h.double(), w2.double(), eps2)) < tol
    assert rel(pd, after) < 3e-6 and torch.equal(pd[[1, 3]].cpu(), prev[[1, 3]])
    # without slots every sequence begins with zeros and nothing is kept
    got, _, none = mix.shift_mix(h.to(DEV), w.to(DEV), eps, DT[dtype], mu.to(DEV), seq, cu, 3)
    assert none is None and rel(got[a], n[a] - n[a] * mu.double()) < tol
    # two norms of the same rows, no sequences
    none, first, other = mix.shift_mix(h.to(DEV), w.to(DEV), eps, DT[dtype], plain=True, second=(w2.to(DEV), eps2))
    assert none is None and torch.equal(first, plain) and torch.equal(other, second)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("T,rank,C", [(1, 1, 5), (7, 16, 96), (8, 64, 200), (9, 5, 33), (300, 24, 128), (130, 100, 40), (150, 8, 1030),
                                      (333, 70, 517), (64, 64, 514), (1, 1000, 6)])
def test_decays_out_of_two_projections(dtype, T, rank, C):
    from rllm_b200.kernels import mix
    wide, w2, b = rnd(T, rank + 8, seed=1, scale=1.5).to(DT[dtype]), rnd(C, rank, seed=2).to(DT[dtype]), rnd(C, seed=3, scale=3.0) - 2
    z = wide[:, 3: 3 + rank]
    want = torch.exp(-torch.exp(torch.tanh(z.double()) @ w2.double().T + b.double()))
    got = mix.lowrank_decay(wide.to(DEV)[:, 3: 3 + rank], w2.T.contiguous().to(DEV), b.to(DEV))
    assert got.dtype == torch.float32 and rel(got, want) < 1e-5 and float(got.min()) >= 0 and float(got.max()) <= 1


@pytest.mark.parametrize("E,top,groups,keep,scale", [(16, 3, 1, 1, 1.0), (12, 3, 4, 2, 2.5), (8, 1, 2, 1, 0.3), (64, 6, 8, 3, 1.7),
                                                     (9, 2, 3, 1, 1.0), (7, 3, 7, 5, 1.5), (200, 8, 4, 2, 4.0), (24, 5, 3, 3, 0.7)])
def test_corrected_router_with_limited_groups(E, top, groups, keep, scale):
    """Choice scores on both sides of zero; groups of one expert; rows longer than the experts; weights from the scores
    without the correction, divided by their sum."""
    from rllm_b200.kernels import mix
    z, c = rnd(37, E + 3, seed=E + top, scale=2.0), torch.rand(E, generator=torch.Generator().manual_seed(E)) * 1.2 - 1.0
    r = {"experts": E, "top": top, "scale": scale}
    if groups > 1:
        r["groups"] = {"count": groups, "keep": keep}
    idx, wt = P.route(z[:, :E].double(), torch.eye(E, dtype=P.DT), c.double(), r)
    gi, gw = mix.moe_topk(z.to(DEV), top, groups, keep, True, "sigmoid", experts=E, correction=c.to(DEV), group_sum=2, sum_eps=1e-20,
                          scale=scale)
    assert torch.equal(gi.cpu().long(), idx) and rel(gw, wt) < 2e-6
    plain, _ = mix.moe_topk(z.to(DEV), top, groups, keep, True, "sigmoid", experts=E)
    if 1 < top < E // 2:
        assert not torch.equal(plain, gi)                     # the correction does move choices here
    if 1 < groups and 1 < keep < groups and E // groups > 2:
        one, _ = mix.moe_topk(z.to(DEV), top, groups, keep, True, "sigmoid", experts=E, correction=c.to(DEV), group_sum=1)
        assert not torch.equal(one, gi)                       # and so does the second of a group's two best


@pytest.mark.parametrize("H", [40, 37, 1024, 4100])
@pytest.mark.parametrize("with_mixer", [True, False])
def test_sum_of_a_layer_with_a_gated_summand(H, with_mixer):
    from rllm_b200.kernels import hybrid
    T = 9
    h, m, parts, shared, z = rnd(T, H, seed=1), rnd(T, H, seed=2), rnd(T, 3, H, seed=3), rnd(T, H, seed=4), rnd(T, 5, seed=5, scale=2.0)
    want = h.double() + parts.double().sum(1) + shared.double() * torch.sigmoid(z[:, 2:3].double())
    want = want + m.double() if with_mixer else want
    hd = h.to(DEV)
    plain = ([m.to(DEV)] if with_mixer else []) + [parts.to(DEV), shared.to(DEV)]
    hybrid.combine(hd, plain=plain, gate=z.to(DEV)[:, 2:])
    assert rel(hd, want) < 2e-6


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("T,G,K,N,last", [(3, 4, 64, 96, 16), (32, 5, 128, 200, 24), (33, 5, 128, 200, 24), (1, 2, 24, 40, 40),
                                          (300, 5, 72, 64, 8), (40, 5, 50, 28, 5), (7, 5, 50, 28, 5), (150, 3, 256, 512, 3), (9, 5, 128, 128, 16),
                                          (50, 5, 192, 256, 64), (300, 5, 64, 128, 40), (2100, 4, 128, 256, 128), (8, 5, 8320, 32, 16),
                                          (700, 5, 1024, 1024, 64)])
def test_products_of_mixes_side_by_side(dtype, T, G, K, N, last):
    """A product per mix, the last of another height: in one launch for steps of few tokens, a product each beyond."""
    from rllm_b200.kernels.backend import Backend
    be = Backend(DT[dtype], DEV)
    x, w = rnd(T, G, K, seed=1).to(DT[dtype]), rnd((G - 1) * N + last, K, seed=2).to(DT[dtype])
    want = torch.cat([x[:, g].double() @ w[g * N: (g + 1) * N].double().T for g in range(G)], 1)
    got = be.linear_mixes(x.to(DEV), w.to(DEV), N)
    assert got.dtype == DT[dtype] and rel(got, want) < (5e-6 if dtype == "float32" else 8e-3)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("T,G,K,N", [(5, 3, 64, 40), (70, 3, 20, 37), (200, 2, 128, 128), (9, 4, 40, 7)])
def test_a_gate_per_output_behind_a_product_per_head(dtype, T, G, K, N):
    from rllm_b200.kernels import mix
    dt = DT[dtype]
    a, w, gate = rnd(T, G * K, seed=1).to(dt), rnd(G, N, K, seed=2).to(dt), rnd(T, G * N + 3, seed=3, scale=2.0).to(dt)
    out = torch.empty(T, G * N, dtype=dt, device=DEV)
    mix.grouped_gemm_uniform(a.to(DEV), K, w.to(DEV), out, N, mix.GEPI_STORE, gate=gate.to(DEV)[:, 3:], gate_cols=True)
    want = torch.cat([a[:, g * K:(g + 1) * K].double() @ w[g].double().T for g in range(G)], 1) * torch.sigmoid(gate[:, 3:].double())
    assert rel(out, want) < (2e-6 if dtype == "float32" else 8e-3)


def test_bounded_logits_and_the_embedding_added_again():
    from rllm_b200.kernels import mix, ops
    x = rnd(7, 1001, seed=1, scale=30.0)
    for cap in (0.5, 8.0, 1e4):
        assert rel(ops.softcap(x.to(DEV).clone(), cap), P.softcap(x.double(), cap)) < 1e-6
    for dtype in DT:
        for H in (24, 300):
            h, v, table = rnd(6, H, seed=2), rnd(H, seed=3), rnd(11, H, seed=4).to(DT[dtype])
            ids = torch.tensor([3, 10, 0, 3, 11, -1], dtype=torch.int32)      # the last two name no row: nothing of the table is added
            want = h.double() + v.double()
            want[:4] += table.double()[ids[:4].long()] * 1.7
            assert rel(mix.add_embedding_row(h.to(DEV), v.to(DEV), ids.to(DEV), table.to(DEV), 1.7), want) < 1e-6


# ------------------------------------------------------------------ time mixing over steps and slots

def wkv_weights(W, H, d, r, seed):
    C = H * d
    shapes = {"r": (C, W), "k": (C, W), "v": (C, W), "g": (C, W), "w1": (r, W), "w2": (C, r), "w0": (C,), "u": (H, d), "norm": (C,),
              "o": (W, C), **{"mu." + s: (W,) for s in "rkvgw"}}
    gen = torch.Generator().manual_seed(seed)
    w = {"x." + k: Z.arrange("mix." + k, rnd(*s, seed=seed + i, scale=0.25), gen) for i, (k, s) in enumerate(shapes.items())}
    w["x.norm"] = w["x.norm"] + 1
    return w


def with_norm(w, W, seed):
    return rnd(W, seed=seed, scale=0.3) + 1


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("W,H,d,r", [(48, 3, 20, 6), (40, 1, 64, 16), (52, 4, 5, 1), (64, 2, 130, 24), (72, 5, 32, 8), (37, 2, 9, 3),
                                     (128, 1, 256, 8)])
def test_time_mixing_over_steps_and_slots(dtype, W, H, d, r):
    """Whole, prefill and single tokens, portions down to two tokens, token by token; the first token, its shift and its
    own (bonus) share count in the yardstick; a request that takes over a slot starts from zero."""
    n, eps = 97, 1e-5
    w, wn = wkv_weights(W, H, d, r, seed=d), with_norm(None, W, 5)
    block = built_block(W, Z.wkv(H, d, r, None), eps)
    part, norm = block.mixer, block.norm
    bind(part, w, dtype, "x.")
    bind(norm, {"norm1": wn}, dtype)
    st = as_stored(w, dtype)
    m = {"heads": H, "dim": d}
    nrm = lambda x: P.rms_norm(x.double(), norm.weight.double().cpu(), eps)
    h = rnd(n, W, seed=9)
    want = P.wkv(nrm(h), st, "", m, eps)
    h0 = nrm(h)
    h0[0] = -h0[0]
    assert rel(P.wkv(h0, st, "", m, eps)[-1:], want[-1:]) > 1e-3             # the first token is still felt by the last one
    no_bonus = dict(st, u=torch.ones_like(st["u"]))
    no_shift = dict(st, **{"mu.v": torch.zeros_like(st["mu.v"])})
    assert rel(P.wkv(nrm(h), no_bonus, "", m, eps), want) > 3e-2 and rel(P.wkv(nrm(h), no_shift, "", m, eps), want) > 3e-2
    hd = h.to(DEV)
    tol = 3e-5 if dtype == "float32" else 3e-2

    def step(hs, entries, spans):
        rows = torch.cat([hd[a:b] for a, b in spans.values()])
        return hs.run(entries, lambda ctx, cache: part.forward_stream(rows, norm, ctx, cache)[0])
    outs = over_schedules(dtype, n, step, lambda: Harness(dtype, [part.cache_spec()], slots=2), want, tol)
    if dtype == "float32":
        assert all(torch.equal(o, outs["whole"]) for o in outs.values())     # no sum's order depends on the cut
    # two requests in one step, unequal portions beside single tokens; then a third in a slot that was used
    hb = rnd(47, W, seed=10)
    want_b = P.wkv(nrm(hb), st, "", m, eps)
    hbd = hb.to(DEV)
    hs = Harness(dtype, [part.cache_spec()], slots=2)
    got_a, got_b, ia, ib = [], [], 0, 0
    for qa, qb in ((30, 5), (1, 1), (65, 39), (1, 2)):
        y = hs.run([("a", qa), ("b", qb)], lambda ctx, cache: part.forward_stream(torch.cat([hd[ia: ia + qa], hbd[ib: ib + qb]]),
                                                                                 norm, ctx, cache)[0])
        got_a.append(y[:qa]); got_b.append(y[qa:])
        ia += qa; ib += qb
    assert rel(torch.cat(got_a), want) < tol and rel(torch.cat(got_b), want_b) < tol
    hs.engine.end(["a", "b"])
    again = hs.run([("c", 47)], lambda ctx, cache: part.forward_stream(hbd, norm, ctx, cache)[0])       # starts from zero
    assert rel(again, want_b) < tol


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("H,d", [(2, 24), (1, 64), (3, 128)])
def test_long_portions_run_in_chunks_side_by_side(dtype, H, d):
    """Portions of 384 tokens and more are cut into chunks whose states are joined: 700 tokens beside 130 and a single one,
    the state carried on into a further long portion and single tokens; the decays slow enough to reach over chunks."""
    W, r, eps = 40, 8, 1e-5
    w, wn = wkv_weights(W, H, d, r, seed=d), with_norm(None, W, 5)
    block = built_block(W, Z.wkv(H, d, r, None), eps)
    part, norm = block.mixer, block.norm
    bind(part, w, dtype, "x.")
    bind(norm, {"norm1": wn}, dtype)
    st, m = as_stored(w, dtype), {"heads": H, "dim": d}
    lens = {"a": 700 + 400 + 3, "b": 130 + 1 + 3, "c": 1 + 385 + 3}
    src = {k: rnd(n, W, seed=20 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: P.wkv(P.rms_norm(x.double(), norm.weight.double().cpu(), eps), st, "", m, eps) for k, x in src.items()}
    hs = Harness(dtype, [part.cache_spec()], slots=3)
    at, got = {k: 0 for k in lens}, {k: [] for k in lens}
    from rllm_b200.parts import gla
    chunks, real = [], gla.scan_chunk
    gla.scan_chunk = lambda ctx, c: (chunks.append(real(ctx, c)), chunks[-1])[1]
    try:
        for st_ in [{"a": 700, "b": 130, "c": 1}, {"a": 400, "b": 1, "c": 385}] + [{"a": 1, "b": 1, "c": 1}] * 3:
            rows = torch.cat([src[k][at[k]: at[k] + q] for k, q in st_.items()]).to(DEV)
            y = hs.run(list(st_.items()), lambda ctx, cache: part.forward_stream(rows, norm, ctx, cache)[0])
            o = 0
            for k, q in st_.items():
                got[k].append(y[o: o + q]); o += q; at[k] += q
    finally:
        gla.scan_chunk = real
    assert chunks == [128, 128, 0, 0, 0]
    for k in lens:
        assert rel(torch.cat(got[k]), want[k]) < (3e-5 if dtype == "float32" else 3e-2), k


# ------------------------------------------------------------------ attention over latents, over steps

def lat_weights(W, m, seed):
    H, d, rot, vd, rank, qr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
    shapes = {"dq": (qr, W), "dq.norm": (qr,), "uq": (H * (d + rot), qr), "dkv": (rank + rot, W), "dkv.norm": (rank,),
              "uk": (H * d, rank), "uv": (H * vd, rank), "g": (H * vd, W), "o": (W, H * vd)}
    w = {"x." + k: rnd(*s, seed=seed + i, scale=0.25) for i, (k, s) in enumerate(shapes.items())}
    w["x.dkv.norm"] = w["x.dkv.norm"] + 1
    w["x.dq.norm"] = w["x.dq.norm"] + 1
    return w


YARN = (4.0, 64, 8.0, 1.0)
LATS = [(Z.lat(3, 24, 16, 40, 30, 48, 0.17, None, (700.0, 16, YARN))["mixer"], 4),
        (Z.lat(2, 16, 8, 16, 56, 24, 0.2, None, (500.0, 6, None))["mixer"], 16),
        (Z.lat(5, 8, 0, 8, 17, 40, 0.3, None)["mixer"], 8),
        (Z.lat(1, 10, 6, 14, 22, 20, 0.25, None, (5000.0, 6, (2.5, 100, 3.0, 0.5)))["mixer"], 8),
        (Z.lat(9, 12, 4, 20, 24, 36, 0.2, None, (100.0, 4, (16.0, 4096, 32.0, 1.0)))["mixer"], 4),
        (Z.lat(16, 32, 32, 48, 64, 128, 0.08, None, (10000.0, 32, YARN))["mixer"], 16),
        (Z.lat(4, 16, 16, 24, 40, 272, 0.08, None, (10000.0, 16, YARN))["mixer"], 8)]


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("m,page", LATS)
def test_latent_attention_with_a_query_latent_and_a_full_gate_over_steps(dtype, m, page):
    """Tokens at a few positions (the first, page borders, far back) are made large in one number of the input, which all their
    keys share: queries that follow see them stand out. Leaving out the scaling of the rotation, the queries'
    norm or one marked token moves the yardstick."""
    W, n, eps = 40, 97, 1e-6
    w = lat_weights(W, m, seed=m["heads"])
    h = rnd(n, W, seed=9)
    marked = {0, 1, page - 1, page, 2 * page + 1, 50}
    for p in marked:
        h[p, 0] += 6.0
    x = h.to(DT[dtype])
    st = as_stored(w, dtype)
    want = P.latent_attention(x.double(), st, "", m, eps)
    for p in (0, page):
        other = x.double().clone()
        other[p, 0] -= 6.0
        assert rel(P.latent_attention(other, st, "", m, eps)[p + 1:], want[p + 1:]) > 3e-3
    if m["rot_dim"] and "scaling" in m["rot"]:
        plain_rot = dict(m, rot={k: v for k, v in m["rot"].items() if k != "scaling"})
        assert rel(P.latent_attention(x.double(), st, "", plain_rot, eps), want) > 1e-3
    block = built_block(W, {"type": "latent_attention", "mixer": m, "mlp": None}, eps)
    part = block.mixer
    assert part.cache_spec().width == m["kv_rank"] + m["rot_dim"]
    bind(part, w, dtype, "x.")
    hd = x.to(DEV)
    tol = 3e-5 if dtype == "float32" else 5e-2

    def step(hs, entries, spans):
        rows = torch.cat([hd[a:b] for a, b in spans.values()])
        return hs.run(entries, lambda ctx, cache: part.forward(rows, ctx, cache))
    outs = over_schedules(dtype, n, step, lambda: Harness(dtype, [part.cache_spec()], page_size=page,
                                                          pages=2 + (n + page - 1) // page), want, tol)
    if dtype == "float32":
        assert all(torch.equal(o, outs["whole"]) for o in outs.values())
    # two requests in one step; then a third on pages that were used
    hb = rnd(47, W, seed=10)
    hb[3, 0] += 6.0
    xb = hb.to(DT[dtype])
    want_b = P.latent_attention(xb.double(), st, "", m, eps)
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


# ------------------------------------------------------------------ feed-forwards and the layer's sum

@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("T", [1, 9, 40, 300])
@pytest.mark.parametrize("W,ff,experts,top,groups,shared", [(64, 48, 8, 3, (4, 2), 80), (40, 20, 6, 2, None, None), (52, 12, 7, 1, None, 10),
                                                            (128, 64, 15, 4, (3, 2), 64), (72, 32, 16, 6, (2, 1), 36)])
def test_routed_experts_with_a_gated_shared_one(dtype, T, W, ff, experts, top, groups, shared):
    """The feed-forward and the sum it ends in. Choices are taken from the package's own router logits where they are
    close calls in 16 bits: the yardstick gets the rounded input, and rows whose choice hangs on a few thousandths are left out."""
    layer = Z.wkv(1, 2, 1, Z.moe(ff, experts, top, 1.6, groups, shared))
    part = built_block(W, layer).ffn
    gen = torch.Generator().manual_seed(T)
    w = {}
    for q in part.walk():
        pre = "x." + ("shared." if q is not part else "")
        for p_ in q.params():
            for i, s in enumerate(p_.sources):
                w[pre + s.name] = Z.arrange("." + s.name, rnd(*s.shape, seed=len(w) + 7, scale=0.25), gen)
    from rllm_b200.weights.loader import storage_dtype
    part.set_prefix("x.")
    for q in part.walk():
        for p_ in q.params():
            t = torch.cat([w[q.prefix + s.name] for s in p_.sources], 0)
            setattr(q, p_.attr, t.to(storage_dtype(p_.role, torch.bfloat16, DT[dtype])).to(DEV).contiguous())
    for q in part.walk():
        q.finalize(torch.device(DEV), DT[dtype])
    st = as_stored({k: v.to(torch.bfloat16) if k == "x.correction" and dtype == "bfloat16" else v for k, v in w.items()}, dtype)
    x = rnd(T, W, seed=3).to(DT[dtype])
    r = layer["mlp"]["router"]
    want = P.moe(x.double(), st, "", layer["mlp"])
    s = torch.sigmoid(x.double() @ st["router"].T) + st["correction"]
    sure = torch.ones(T, dtype=torch.bool)
    for eps in (3e-3, -3e-3):                       # the same choice with every second expert's score moved a little
        moved = st["correction"].clone()
        moved[::2] += eps
        sure &= (P.route(x.double(), st["router"], moved, r)[0].sort(-1).values ==
                 P.route(x.double(), st["router"], st["correction"], r)[0].sort(-1).values).all(-1)
    assert s.min() < 0 < s.max() and int(sure.sum()) >= 0.6 * T
    hs = Harness(dtype, [])

    class Ctx:
        backend = hs.backend
    y = part.forward(x.to(DEV), Ctx, None)
    h = torch.zeros(T, W, device=DEV)
    hs.backend.combine(h, torch.zeros(T, W, device=DEV), y)
    got = h.cpu()
    tol = 2e-5 if dtype == "float32" else 2.5e-2
    keep = torch.ones_like(sure) if dtype == "float32" else sure
    assert rel(got[keep], want[keep]) < tol
    if shared:
        ungated = want + P.gated(x.double(), st, "shared.") * (1 - torch.sigmoid(x.double() @ st["shared.sg"].T))
        assert rel(ungated, want) > 1e-2


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("T", [5, 70, 200])
@pytest.mark.parametrize("layer", [Z.lat(3, 24, 16, 40, 30, 48, 0.3, Z.dense(72), (700.0, 16, YARN)), Z.wkv(3, 20, 8, Z.dense(56)),
                                   Z.lat(2, 12, 4, 20, 12, 12, 0.3, None, (77.0, 4, None)), Z.wkv(2, 16, 4, None)])
def test_mixer_and_feed_forward_read_norms_of_the_same_stream(dtype, T, layer):
    """A layer alone: two norms with weights far apart, both of the stream before the layer."""
    W, eps = 64, 1e-3
    block = built_block(W, layer, eps)
    block.set_prefix("")
    gen = torch.Generator().manual_seed(3)
    from rllm_b200.weights.loader import storage_dtype
    w = {}
    for q in block.walk():
        for p_ in q.params():
            for s in p_.sources:
                w[q.prefix + s.name] = Z.arrange(q.prefix + s.name, rnd(*s.shape, seed=len(w) + 7, scale=0.2), gen)
                if s.init == "norm":
                    w[q.prefix + s.name] += 2.0 if s.name == "norm2" else 1.0
            setattr(q, p_.attr, torch.cat([w[q.prefix + s.name] for s in p_.sources], 0).to(
                storage_dtype(p_.role, torch.bfloat16, DT[dtype])).to(DEV).contiguous())
    for q in block.walk():
        q.finalize(torch.device(DEV), DT[dtype])
    st = {k: (v.to(torch.bfloat16) if dtype == "bfloat16" else v).double() for k, v in w.items()}
    h = rnd(T, W, seed=4, scale=0.5)
    mixer = P.MIXERS[layer["type"]](P.rms_norm(h.double(), st["norm1"], eps), st, "mix.", layer["mixer"], eps)
    want = mixer if layer["mlp"] is None else mixer + P.dense(P.rms_norm(h.double(), st["norm2"], eps), st, "mlp.", layer["mlp"])
    hs = Harness(dtype, [block.cache_spec()], page_size=8, pages=40)
    hd = h.to(DEV)
    hs.run([("a", T)], lambda ctx, cache: block.forward(hd, ctx, cache))
    assert rel(hd - h.to(DEV), want) < (3e-5 if dtype == "float32" else 3e-2)


# ------------------------------------------------------------------ whole models

def requests_for(name, lens=(9, 61, 23, 150, 37, 2)):
    vocab = Z.TINY[name][0]["vocab"]
    return {f"r{i}": Z.random_prompt(n, vocab, 100 * len(name) + ord(name[1]) + i) for i, n in enumerate(lens)}


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("zufotar")
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
ROUTED = {n for n, (c, *_) in Z.TINY.items() if any((L["mlp"] or {}).get("kind") == "moe" for L in c["layers"])}


def allowed(name):
    """The share of positions that may lie off in bfloat16: a token whose router met a close call has another expert, and
    the head norm behind the recurrence makes much of a first token whose own share is nearly nothing."""
    return 0.25 if name in ROUTED else 0.02


def engine_for(dirs, name, dtype, steps, reqs, max_requests=3):
    from rllm_b200.engine import load_engine
    return load_engine(dirs[name], dtype=dtype, page_size=Z.TINY[name][3],
                       max_tokens=replay.max_live_tokens(steps, reqs), max_requests=max_requests)


@pytest.mark.parametrize("name", list(Z.TINY))
def test_residual_stream_after_every_layer_run(dirs, name):
    """In float32, layer run by layer run (every pass of a loop): the first one that differs names the mechanism."""
    from rllm_b200.engine import Entry, load_engine
    from rllm_b200.parts import LoopStep
    cfg, w = P.read_model_dir(dirs[name])
    toks = Z.random_prompt(45, cfg["vocab"], 9)
    _, kept = P.forward(cfg, w, toks, keep_layers=True)
    eng = load_engine(dirs[name], dtype="float32", page_size=Z.TINY[name][3], max_tokens=64, max_requests=1)
    got = []
    for b in eng.model.blocks:
        if isinstance(b, LoopStep):
            continue

        def wrap(h, ctx, cache, f=b.forward):
            out = f(h, ctx, cache)
            got.append(h.detach().float().cpu().clone())
            return out
        b.forward = wrap
    eng.step([Entry("a", toks, [])])
    runs = P.layer_runs(cfg)
    assert len(got) == len(kept) == len(runs)
    for i, (g, k) in enumerate(zip(got, kept)):
        assert rel(g, k) < 5e-5, f"{name}: the stream differs after layer run {i} ({cfg['layers'][runs[i][0]]['type']})"


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
        check(got, plain[name], 3e-4, f"{name} float32 {family}")
    else:
        check(got, plain[name], 8e-2, f"{name} bfloat16 {family}", allow=allowed(name))


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
            assert worst <= 3e-5, f"{name} {family}: differs from whole prompts by {worst}"


@pytest.mark.parametrize("name", ["UA", "UC", "UD"])
@pytest.mark.parametrize("dtype,tol", [("float32", 3e-4), ("bfloat16", 8e-2)])
def test_long_decoding_through_graphs(dirs, name, dtype, tol):
    """Two requests decoded side by side for 120 steps from prompts of 3 and 30 tokens: states and last rows are carried
    through replayed graphs, latents of decoded tokens fill page after page."""
    from rllm_b200.engine import Entry, load_engine
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
    check(got, {(k, i): want[k][i] for (k, i) in got}, tol, f"long decoding {name} {dtype}",
          allow=0.0 if dtype == "float32" else allowed(name))


@pytest.mark.parametrize("name", ["UF", "UG"])
@pytest.mark.parametrize("dtype", list(DT))
def test_long_prompts_in_portions_and_decoding(dirs, name, dtype):
    """Prompts of 1,320 and 720 tokens in portions of 600 (the chunked recurrence, products of long portions) and single
    tokens; on pages and slots that went back to the pool. Models without a choice of experts (one chooses all it has), so
    that every position counts."""
    from rllm_b200.engine import Entry, load_engine
    cfg, w = P.read_model_dir(dirs[name])
    toks = {"x": Z.random_prompt(1320, cfg["vocab"], 5), "y": Z.random_prompt(720, cfg["vocab"], 6)}
    want = {k: P.forward(cfg, w, t).numpy() for k, t in toks.items()}
    eng = load_engine(dirs[name], dtype=dtype, page_size=16, max_tokens=1344, max_requests=1)
    for rid in ("y", "x"):
        t, got, i, n = toks[rid], {}, 0, len(toks[rid])
        for q in [600] * ((n - 20) // 600) + [(n - 20) % 600] + [1] * 20:
            lg = eng.step([Entry(rid, t[i: i + q], [0, q - 1] if q > 1 else [0])]).float().cpu().numpy()
            got[(rid, i)] = lg[0]
            got[(rid, i + q - 1)] = lg[-1]
            i += q
        eng.end([rid])
        eng.check()
        check(got, {k: want[rid][k[1]] for k in got}, 3e-4 if dtype == "float32" else 8e-2, f"long prompt {rid}",
              allow=0.0 if dtype == "float32" else 0.05)


@pytest.mark.parametrize("name", ["UB", "UC", "UE", "UF"])
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
    name = "UA"
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
    check(got, {(i, p): want[i][p] for (i, p) in got}, 3e-4, "padded graph")


def test_command_line_runs_the_design(dirs):
    name = "UF"
    cfg, w = P.read_model_dir(dirs[name])
    prompt = Z.random_prompt(11, cfg["vocab"], 3)
    toks = prompt + P.greedy(cfg, w, prompt, 5)
    r = subprocess.run([sys.executable, os.path.join(replay.ROOT, "bin", "rllm"), "run", "--model", dirs[name],
                        "--prompt-ids", " ".join(map(str, prompt)), "--max-tokens", "5", "--temperature", "0",
                        "--dtype", "float32", "--kv-pages", "32"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.split()] == toks[len(prompt):]


@pytest.mark.parametrize("name,dtype", [("UA", "float32"), ("UD", "bfloat16")])
def test_trace_program_runs_the_design(dirs, plain, tmp_path, name, dtype):
    reqs = requests_for(name)
    steps = replay.mixed(reqs, max_live=4)
    got = replay.run_program(dirs[name], dtype, steps, str(tmp_path / "out"), replay.max_live_tokens(steps, reqs),
                             Z.TINY[name][0]["vocab"], extra_args=["--page-size", "16"])
    if dtype == "float32":
        check(got, plain[name], 3e-4, "trace program")
    else:
        check(got, plain[name], 8e-2, "trace program bfloat16", allow=allowed(name))
