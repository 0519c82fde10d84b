"""Zufotar without a GPU: the configuration reader, the registry, the tensors the model expects, its cache layers and its
schedule, and the plain implementation's own mechanisms against closed forms."""
import json

import pytest
import torch

import plain_zufotar as P
import zufotar_tiny as Z


def test_registry_finds_the_design_by_its_architecture_string():
    from rllm_b200.config import config_from_dict, registered_architectures
    assert "Zufotar" in registered_architectures()
    arch, cfg = config_from_dict(Z.UA)
    assert arch.name == "Zufotar" and (cfg.width, cfg.vocab, cfg.norm_eps, cfg.embedding_scale) == (88, 150, 1e-5, 0.7)
    assert cfg.logit_softcap == 2.0 and (cfg.loop_start, cfg.loop_stop, cfg.loop_times) == (1, 3, 2)
    a, r = cfg.layers[0], cfg.layers[1]
    m = a.mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale) == (3, 24, 16, 40, 56, 48, 0.3)
    assert (m.rot_base, m.rot_dims) == (700.0, 16) and m.rot_scaling.to_dict() == {"factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 1.0}
    assert a.mlp.kind == "dense" and a.mlp.ff == 72
    assert (r.type, r.mixer.heads, r.mixer.dim) == ("wkv", 4, 20)
    f = r.mlp
    assert (f.kind, f.ff, f.experts, f.top, f.scale, f.groups, f.keep, f.shared_ff) == ("moe", 24, 8, 3, 1.7, 4, 2, 40)
    assert cfg.layers[3].mlp is None
    assert cfg.layer_runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    for raw in (Z.UA, Z.UB, Z.UC, Z.UD, Z.UE, Z.UF, Z.UG):
        c = config_from_dict(raw)[1]
        assert type(c).from_dict(c.to_dict()) == c and c.layer_runs() == P.layer_runs(raw)
    _, cb = config_from_dict(Z.UB)            # what a configuration leaves out does not exist
    assert cb.logit_softcap is None and not cb.has_loop and cb.layers[0].mixer.rot_scaling is None
    assert cb.layers[0].mlp.shared_ff is None and cb.layers[1].mixer.rot_dim == 0 and cb.layers[2].mlp is None


@pytest.mark.parametrize("spoil,what", [
    (lambda c: c["layers"][0].update(type="gla"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][1]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=5), "groups"),
    (lambda c: c["layers"][1]["mlp"].update(kind="glu"), "kind"),
    (lambda c: c["layers"][0].update(mlp=3), "mlp"),
    (lambda c: c.update(logit_softcap=0.0), "logit_softcap"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c.pop("embedding"), "embedding"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_a_configuration_that_cannot_be_is_refused(spoil, what):
    from rllm_b200.config import ConfigError, config_from_dict
    raw = json.loads(json.dumps(Z.UA))
    spoil(raw)
    with pytest.raises(ConfigError) as e:
        config_from_dict(raw)
    assert what in str(e.value)


def test_cache_layers_and_schedule():
    """Every run of a layer has pages or a state of its own; a pass begins with its vector, all but the first with the
    embedding again."""
    from rllm_b200.config import config_from_dict
    from rllm_b200.parts import LatentCacheSpec, LoopStep, StateSpec
    arch, cfg = config_from_dict(Z.UA)
    m = arch.build(cfg)
    specs = m.cache_specs()
    assert [type(s) for s in specs] == [LatentCacheSpec, StateSpec, LatentCacheSpec, StateSpec, LatentCacheSpec, StateSpec]
    assert specs[0].width == 64 and specs[2].width == 44 and specs[0].window is None
    assert specs[1].tensors == (("S", (4, 20, 20), torch.float32), ("prev", (88,), torch.float32))
    assert [(c.block, c.cache_layer) for c in m.schedule] == [(0, 0), (4, -1), (1, 1), (2, 2), (5, -1), (1, 3), (2, 4), (3, 5)]
    steps = m.blocks[4:]
    assert all(isinstance(s, LoopStep) for s in steps) and [s.embedding is not None for s in steps] == [False, True]
    assert [len(s.params()) for s in steps] == [1, 0]
    assert m.blocks[3].ffn is None and m.blocks[3].ffn_norm is None and m.head.softcap == 2.0
    arch, cfg = config_from_dict(Z.UC)
    assert all(isinstance(s, StateSpec) for s in arch.build(cfg).cache_specs())


def test_expected_tensors(tmp_path):
    from rllm_b200.config import config_from_dict
    from rllm_b200.weights import WeightError, expected_tensors, load_weights
    arch, cfg = config_from_dict(Z.UA)
    names = {n: tuple(s.shape) for n, s, _, _ in expected_tensors(arch.build(cfg))}
    W = 88
    assert names["embed"] == (150, W) and names["final.norm"] == (W,) and names["loop.step"] == (2, W)
    assert not any(n.startswith("head") for n in names)
    assert names["l0.norm1"] == names["l0.norm2"] == (W,) and names["l0.mlp.up"] == (72, W) and names["l0.mlp.down"] == (W, 72)
    assert names["l0.mix.dq"] == (56, W) and names["l0.mix.dq.norm"] == (56,) and names["l0.mix.uq"] == (120, 56)
    assert names["l0.mix.dkv"] == (64, W) and names["l0.mix.dkv.norm"] == (48,) and names["l0.mix.uk"] == (72, 48)
    assert names["l0.mix.uv"] == (120, 48) and names["l0.mix.g"] == (120, W) and names["l0.mix.o"] == (W, 120)
    for s in "rkvgw":
        assert names[f"l1.mix.mu.{s}"] == (W,)
    for s in "rkvg":
        assert names[f"l1.mix.{s}"] == (80, W)
    assert names["l1.mix.w1"] == (12, W) and names["l1.mix.w2"] == (80, 12) and names["l1.mix.w0"] == (80,)
    assert names["l1.mix.u"] == (4, 20) and names["l1.mix.norm"] == (80,) and names["l1.mix.o"] == (W, 80)
    assert names["l1.mlp.router"] == (8, W) and names["l1.mlp.correction"] == (8,) and names["l1.mlp.shared.sg"] == (1, W)
    assert names["l1.mlp.e7.gate"] == (24, W) and names["l1.mlp.e7.down"] == (W, 24) and names["l1.mlp.shared.up"] == (40, W)
    assert "l3.norm2" not in names and not any(n.startswith("l3.mlp") for n in names)
    assert not any("shared" in n or ".g" == n[-2:] and "mlp" in n for n, *_ in expected_tensors(config_from_dict(Z.UB)[0].build(config_from_dict(Z.UB)[1])))
    d = Z.make_model_dir(tmp_path, "UA")
    # the inner size of the decays is the checkpoint's where the configuration does not give it
    raw = json.loads(open(d + "/config.json").read())
    for L in raw["layers"]:
        L["mixer"].pop("decay_rank", None)
    arch2, cfg2 = config_from_dict(raw)
    model = arch2.build(cfg2)
    load_weights(model, d, torch.float32, torch.device("cpu"))
    w = P.read_model_dir(d)[1]
    assert set(w) == set(names)
    moe = model.blocks[1].ffn                   # the shared expert's gate stands under the router's rows, then zeros
    assert moe.w_router.shape == (16, W) and torch.equal(moe.w_router[8], w["l1.mlp.shared.sg"][0].float())
    assert torch.equal(moe.w_router[:8], w["l1.mlp.router"].float()) and float(moe.w_router[9:].abs().max()) == 0
    mix = model.blocks[1].mixer
    assert mix._rank == 12 and torch.equal(mix._mu[4], w["l1.mix.mu.w"].float())
    assert torch.equal(mix.w_in[320:], w["l1.mix.w1"].float()) and torch.equal(mix.w_in[80:160], w["l1.mix.k"].float())
    raw["layers"][1]["mixer"]["heads"] = 2
    arch3, cfg3 = config_from_dict(raw)
    with pytest.raises(WeightError):
        load_weights(arch3.build(cfg3), d, torch.float32, torch.device("cpu"))


def test_random_weights_need_the_inner_size_of_the_decays(tmp_path):
    from rllm_b200.weights import write_random_model
    raw = json.loads(json.dumps(Z.UF))
    raw["layers"][0]["mixer"].pop("decay_rank")
    with pytest.raises(ValueError, match="w1"):
        write_random_model(raw, 1, str(tmp_path / "x"))


def test_plain_mechanisms_against_closed_forms():
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=P.DT)
    # the recurrence with decays of one and a bonus of one adds up every pair of tokens like attention without softmax
    q, k, v = r(6, 2, 5), r(6, 2, 5), r(6, 2, 5)
    one = torch.ones(6, 2, 5, dtype=P.DT)
    o, S = P.wkv_steps(q, k, v, one, one[0])
    s = torch.einsum("ihd,jhd->hij", q, k).tril()
    assert torch.allclose(o, torch.einsum("hij,jhd->ihd", s, v)) and torch.allclose(S, torch.einsum("jhk,jhv->hkv", k, v))
    # without a bonus a token does not read itself; a decay acts on what later tokens read, not on the token's own
    o0, _ = P.wkv_steps(q, k, v, one, 0 * one[0])
    assert torch.allclose(o0, torch.einsum("hij,jhd->ihd", s.tril(-1), v))
    half, _ = P.wkv_steps(q[:3], k[:3], v[:3], 0.5 * one[:3], one[0])
    w = torch.tensor([[1, 0, 0], [1, 1, 0], [0.5, 1, 1]], dtype=P.DT)
    assert torch.allclose(half, torch.einsum("hij,jhd->ihd", s[:, :3, :3] * w, v[:3]))
    # a run in two halves with the state handed on is the whole run
    a, Sa = P.wkv_steps(q[:4], k[:4], v[:4], 0.7 * one[:4], 2 * one[0])
    b, _ = P.wkv_steps(q[4:], k[4:], v[4:], 0.7 * one[4:], 2 * one[0], Sa)
    assert torch.allclose(torch.cat([a, b]), P.wkv_steps(q, k, v, 0.7 * one, 2 * one[0])[0])
    # the token shift: shares of 0 leave the rows, shares of 1 give the row before, zeros before the first
    x = r(5, 3)
    assert torch.equal(P.token_shift(x, torch.zeros(3, dtype=P.DT)), x)
    y = P.token_shift(x, torch.ones(3, dtype=P.DT))
    assert torch.allclose(y[1:], x[:-1]) and float(y[0].abs().max()) == 0
    assert torch.allclose(P.token_shift(x[2:], torch.ones(3, dtype=P.DT), x[1])[0], x[1])
    # routing: the correction moves the choice and not the weights; a group counts by its two best, also when negative
    z = torch.tensor([[2.0, -3.0, 0.5, 0.4, -1.0, -2.0]], dtype=P.DT)
    eye, c = torch.eye(6, dtype=P.DT), torch.full((6,), -5.0, dtype=P.DT)
    idx, wt = P.route(z, eye, c, {"top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 1}})
    assert sorted(idx[0].tolist()) == [2, 3]                   # 0.88 + 0.05 < 0.62 + 0.60
    s = torch.sigmoid(z[0])
    assert torch.allclose(wt[0], s[idx[0]] / s[idx[0]].sum() * 3.0)
    c[5] = 0.0
    idx, wt = P.route(z, eye, c, {"top": 1, "scale": 1.0})
    assert idx[0].tolist() == [5] and float(wt[0, 0]) == pytest.approx(1.0)
    # a bound bounds and hardly moves small logits
    t = torch.tensor([1e-3, 1e6], dtype=P.DT)
    assert float(P.softcap(t, 4.0)[1]) == pytest.approx(4.0) and abs(float(P.softcap(t, 4.0)[0]) - 1e-3) < 1e-9
    assert P.softcap(t, None) is t


def test_a_loop_adds_the_embedding_before_every_pass_but_the_first():
    """A model whose layers give nothing: what is left is embedding, vectors and the repeated embedding."""
    cfg = Z.model(5, 4, 2.0, 1e-6, None, (0, 1, 3), [Z.wkv(1, 2, 1, None)])
    g = torch.Generator().manual_seed(2)
    r = lambda *s: torch.randn(*s, generator=g, dtype=P.DT)
    w = {"embed": r(5, 4), "loop.step": r(3, 4), "final.norm": torch.ones(4, dtype=P.DT), "l0.norm1": torch.ones(4, dtype=P.DT)}
    for n, shape in {"r": (2, 4), "k": (2, 4), "v": (2, 4), "g": (2, 4), "w1": (1, 4), "w2": (2, 1), "w0": (2,), "u": (1, 2),
                     "norm": (2,)}.items():
        w["l0.mix." + n] = r(*shape)
    for s in "rkvgw":
        w["l0.mix.mu." + s] = r(4)
    w["l0.mix.o"] = torch.zeros(4, 2, dtype=P.DT)
    _, kept = P.forward(cfg, w, [3, 1], keep_layers=True)
    x0 = w["embed"][[3, 1]] * 2.0
    assert torch.allclose(kept[0], x0 + w["loop.step"][0])
    assert torch.allclose(kept[2], 3 * x0 + w["loop.step"].sum(0))
