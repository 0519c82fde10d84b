"""Danonex without a GPU: the configuration reader, the registry, the tensors the model expects, its cache layers, the
yarn rule of the rotation, and the plain implementation's own mechanisms against closed forms."""
import json
import math

import pytest
import torch

import danonex_tiny as Z
import plain_danonex as P


def test_registry_finds_the_design_by_its_architecture_string():
    from rllm_b200.config import config_from_dict, registered_architectures
    assert "Danonex" in registered_architectures()
    arch, cfg = config_from_dict(Z.DA)
    assert arch.name == "Danonex" and cfg.width == 72 and cfg.vocab == 130 and cfg.norm_eps == 1e-5
    assert cfg.residual_mult == 0.7 and cfg.logit_scale == 1.5
    a, d = cfg.layers[0], cfg.layers[1]
    assert a.type == "attention" and (a.mixer.heads, a.mixer.kv_heads, a.mixer.dim, a.mixer.vdim) == (4, 2, 24, 40)
    assert a.mixer.scale == 0.4 and a.mixer.softcap == 3.0 and a.mixer.rot_dims == 16 and a.mixer.rot_base == 800.0 and a.ff == 96
    s = a.mixer.rot_scaling
    assert (s.factor, s.original, s.fast, s.slow) == (4.0, 64.0, 8.0, 1.0)
    assert d.type == "delta" and (d.mixer.heads, d.mixer.kv_heads, d.mixer.dim, d.mixer.vdim, d.mixer.conv) == (4, 2, 24, 16, 4)
    assert d.ff is None
    assert type(cfg).from_dict(cfg.to_dict()) == cfg
    _, cb = config_from_dict(Z.DB)            # what a configuration leaves out does not exist
    m = cb.layers[0].mixer
    assert m.softcap is None and m.rot_dims == 0 and cb.layers[1].mixer.rot_scaling is None and cb.layers[1].ff is None
    assert type(cb).from_dict(cb.to_dict()) == cb


@pytest.mark.parametrize("spoil,what", [
    (lambda c: c["layers"][0].update(type="ssm"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rotated"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=48), "rotated"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=-1.0), "factor"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "kind"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_a_configuration_that_cannot_be_is_refused(spoil, what):
    from rllm_b200.config import ConfigError, config_from_dict
    raw = json.loads(json.dumps(Z.DA))
    spoil(raw)
    with pytest.raises(ConfigError) as e:
        config_from_dict(raw)
    assert what in str(e.value)


def test_cache_layers_pages_and_states():
    from rllm_b200.config import config_from_dict
    from rllm_b200.parts import KVCacheSpec, StateSpec
    arch, cfg = config_from_dict(Z.DA)
    m = arch.build(cfg)
    specs = m.cache_specs()
    assert [type(s) for s in specs] == [KVCacheSpec, StateSpec, KVCacheSpec, StateSpec]
    assert specs[0] == KVCacheSpec(kv_heads=2, head_dim=24, v_dim=40)
    assert specs[1].tensors == (("S", (4, 24, 16), torch.float32), ("tail", (3, 2 * 48 + 64), torch.float32))
    assert [b.alpha for b in m.blocks] == [0.7] * 4 and m.blocks[1].ffn is None
    arch, cfg = config_from_dict(Z.DC)
    assert all(isinstance(s, StateSpec) for s in arch.build(cfg).cache_specs())


def test_expected_tensors(tmp_path):
    from rllm_b200.config import config_from_dict
    from rllm_b200.weights import WeightError, expected_tensors, load_weights
    arch, cfg = config_from_dict(Z.DA)
    names = {n: tuple(s.shape) for n, s, _, _ in expected_tensors(arch.build(cfg))}
    W = 72
    assert names["embed"] == (130, W) and names["final.norm"] == (W,) and not any(n.startswith("head") for n in names)
    assert names["l0.mix.q"] == (96, W) and names["l0.mix.k"] == (48, W) and names["l0.mix.v"] == (80, W)
    assert names["l0.mix.q.norm"] == (96,) and names["l0.mix.k.norm"] == (48,) and names["l0.mix.sink"] == (4,)
    assert names["l0.mix.o"] == (W, 160) and names["l0.mlp.up"] == (96, W) and names["l0.norm2"] == (W,)
    assert names["l1.mix.q"] == (48, W) and names["l1.mix.v"] == (64, W) and names["l1.mix.v.conv"] == (64, 4)
    assert names["l1.mix.a"] == names["l1.mix.b"] == (4, W) and names["l1.mix.dt_bias"] == names["l1.mix.A_log"] == (4,)
    assert names["l1.mix.g"] == (64, W) and names["l1.mix.norm"] == (16,) and names["l1.mix.o"] == (W, 64)
    assert "l1.norm2" not in names and not any(n.startswith("l1.mlp") for n in names)
    d = Z.make_model_dir(tmp_path, "DA")
    model = arch.build(cfg)
    load_weights(model, d, torch.float32, torch.device("cpu"))
    p = P.read_model_dir(d)[1]
    assert set(p) == set(names)
    # the factor on the logits is folded into the final norm's weight, in float
    assert torch.equal(model.head.norm.weight, p["final.norm"].float() * 1.5)
    raw = json.loads(open(d + "/config.json").read())
    raw["layers"][1]["mixer"]["heads"] = 2
    arch2, cfg2 = config_from_dict(raw)
    with pytest.raises(WeightError):
        load_weights(arch2.build(cfg2), d, torch.float32, torch.device("cpu"))


YARNS = [   # (base, dims, (factor, original, fast, slow))
    (800.0, 16, (4.0, 64, 8.0, 1.0)), (10000.0, 64, (8.0, 4096, 32.0, 1.0)), (100.0, 16, (2.5, 100, 3.0, 0.5)),
    (50.0, 8, (16.0, 4096, 32.0, 1.0)),         # the last frequency still turns often: nothing is divided
    (1e6, 32, (2.0, 8, 4.0, 1.0)),              # the first index falls below 0
    (5000.0, 80, (1.0, 128, 4.0, 4.0)),         # a factor of 1; fast = slow
    (2.0, 6, (3.0, 6.5, 1.0, 0.01)),            # the last index is cut off at dims - 1
]


@pytest.mark.parametrize("base,dims,s", YARNS)
def test_yarn_frequencies_and_magnitude(base, dims, s):
    from rllm_b200.config.danonex import YarnScaling
    from rllm_b200.parts import InterleavedRotary, inverse_frequencies
    sc = YarnScaling(*map(float, s))
    rot = {"base": base, "dims": dims, "scaling": dict(zip(("factor", "original", "fast", "slow"), s))}
    f0 = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=P.DT)
    want, mag = P.yarn(f0, rot)
    assert torch.allclose(torch.tensor(inverse_frequencies(dims, base, sc), dtype=P.DT), want, rtol=1e-13)
    part = InterleavedRotary(dims + 4, base, dims, sc)
    part.finalize(torch.device("cpu"), torch.float32)
    assert part.rotated == dims and abs(part.mag - mag) < 1e-12 and part.inv_freq.dtype == torch.float32
    assert part.mag == pytest.approx(0.1 * math.log(s[0]) + 1)
    # between "as they are" and "all divided"
    assert bool((want <= f0 * (1 + 1e-12)).all()) and bool((want >= f0 / s[0] * (1 - 1e-12)).all())


def test_the_half_split_rotation_takes_the_same_rules():
    from rllm_b200.config.danonex import YarnScaling
    from rllm_b200.parts import RotaryEmbedding
    sc = YarnScaling(4.0, 64.0, 8.0, 1.0)
    part = RotaryEmbedding(24, 800.0, sc, rot_dim=16)
    part.finalize(torch.device("cpu"), torch.float32)
    assert part.rotated == 16 and not part.interleaved and part.mag == pytest.approx(0.1 * math.log(4.0) + 1)
    plain = RotaryEmbedding(24, 800.0, None, rot_dim=16)
    plain.finalize(torch.device("cpu"), torch.float32)
    assert plain.mag == 1.0 and plain.table_key != part.table_key


def test_plain_mechanisms_against_closed_forms():
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=P.DT)
    # a delta rule without decay, with steps of one and orthonormal keys, stores and returns the values
    k = torch.eye(5, dtype=P.DT)[:, None, :]
    v = r(5, 1, 3)
    one = torch.ones(5, 1, dtype=P.DT)
    q = k.roll(1, 0).clone()                     # token t asks for key t - 1 (token 0 for a key that comes later)
    o = P.delta_steps(q, k, v, one, one)
    assert torch.allclose(o[1:, 0], v[:-1, 0]) and float(o[0].abs().max()) == 0.0
    # what a token writes it also reads; a second write to the same key replaces the first
    assert torch.allclose(P.delta_steps(k, k, v, one, one), v)
    k2 = k[[0, 0]]
    assert torch.allclose(P.delta_steps(k2, k2, v[:2], one[:2], one[:2]), v[:2])
    # with decay g the first write is felt as g at the next token
    o = P.delta_steps(k[[0, 0]], k[[0, 1]], v[:2], 0.25 * one[:2], one[:2])
    assert torch.allclose(o[1, 0], 0.25 * v[0, 0])
    # a convolution whose last column alone is set passes the current input on
    w = torch.zeros(4, 3, dtype=P.DT)
    w[:, 2] = 1.0
    x = r(6, 4)
    assert torch.allclose(P.causal_conv(x, w), P.silu(x))
    w = torch.zeros(4, 3, dtype=P.DT)
    w[:, 0] = 1.0
    y = P.causal_conv(x, w)
    assert float(y[:2].abs().max()) == 0.0 and torch.allclose(y[2:], P.silu(x[:-2]))
    # an interleaved rotation keeps lengths (without scaling), is relative in its scores, and turns (1, 0) into (cos, sin)
    rot = {"base": 30.0, "dims": 6}
    a, b = r(1, 2, 8), r(1, 2, 8)
    at = lambda z, p: P.rotate_interleaved(z, rot, torch.tensor([p]))
    assert torch.allclose(at(a, 7).norm(dim=-1), a.norm(dim=-1))
    assert torch.allclose((at(a, 9) * at(b, 4)).sum(-1), (at(a, 25) * at(b, 20)).sum(-1))
    e = torch.zeros(1, 1, 8, dtype=P.DT)
    e[..., 2] = 1.0
    t = at(e, 5)[0, 0]
    ang = 5 * 30.0 ** (-2 / 6)
    assert abs(float(t[2]) - math.cos(ang)) < 1e-12 and abs(float(t[3]) - math.sin(ang)) < 1e-12 and float(t.abs().sum()) < 2.0
    # a sink of the size of the only score halves its weight; a bound bounds and hardly moves small scores
    assert float(P.sink_softmax(torch.full((1, 1, 1), 0.7, dtype=P.DT), torch.ones(1, 1, dtype=torch.bool), torch.tensor([0.7], dtype=P.DT))) == pytest.approx(0.5)
    s = torch.tensor([1e-3, 1.0, 1e6], dtype=P.DT)
    assert torch.allclose(P.capped(s, 4.0)[2], torch.tensor(4.0, dtype=P.DT)) and float((P.capped(s, 4.0)[0] - s[0]).abs()) < 1e-9
    assert P.capped(s, None) is s
    z = torch.linspace(-3, 3, 13, dtype=P.DT)
    assert torch.allclose(P.gelu_erf(z) - P.gelu_erf(-z), z) and float(P.gelu_erf(torch.tensor(10.0, dtype=P.DT))) == pytest.approx(10.0)
