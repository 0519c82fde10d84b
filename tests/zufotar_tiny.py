"""The tests' own small Zufotar configurations and model folders. They differ from each other in every size and option:
head counts, plain / rotated / value sizes, ranks of both latents, a rotation of a part of the rotated vector, of all of it and
none, with the yarn rule (ramps inside the vector, cut off at either end, of no width) and without, experts with and
without groups, a shared expert or none, weights of the experts scaled up, down and not at all, dense feed-forwards and none,
recurrent heads narrower and wider than a warp, bounds of the logits that bite, that hardly do and none, loops of one to
three passes at the start, inside and at the end, and no loop, models of one kind of layer, and of one layer.

Weights that random numbers of one size would leave without effect are drawn on their own: the shares of the token shift
between 0 and 1, decays slow on half the channels, a bonus of about one, router rows large enough to tell experts apart."""
import os

import torch


def lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mlp, rot=None):
    """rot: (base, dims, None or (factor, original, fast, slow)); None: no rotated part"""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if rot[2] is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def wkv(heads, dim, decay_rank, mlp):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "decay_rank": decay_rank}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, scale, groups=None, shared=None):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def model(vocab, width, emb, eps, softcap, loop, layers):
    c = {"architecture": "Zufotar", "vocab": vocab, "width": width, "embedding": {"scale": emb}, "norm": {"eps": eps},
         "layers": layers}
    if softcap is not None:
        c["logit_softcap"] = softcap
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


UA = model(150, 88, 0.7, 1e-5, 2.0, (1, 3, 2), [      # both kinds, every option, a loop inside; a bound that bites
    lat(3, 24, 16, 40, 56, 48, 0.3, dense(72), (700.0, 16, (4.0, 64, 8.0, 1.0))),
    wkv(4, 20, 12, moe(24, 8, 3, 1.7, (4, 2), 40)),
    lat(2, 16, 8, 12, 20, 36, 0.35, moe(32, 6, 2, 0.6, None, 16), (100.0, 6, (2.5, 100, 3.0, 0.5))),
    wkv(2, 44, 8, None),
])
UB = model(200, 64, 1.0, 3e-6, None, None, [          # attention only; no bound, no loop, no scaling, no rotated part
    lat(5, 8, 24, 8, 16, 40, 0.4, moe(16, 4, 1, 1.0, (2, 1)), (100.0, 24, None)),
    lat(2, 20, 0, 32, 48, 24, 0.3, dense(40)),
    lat(1, 12, 12, 20, 8, 16, 0.5, None, (50.0, 12, (16.0, 4096, 32.0, 1.0))),
])
UC = model(90, 52, 2.5, 1e-6, 5.0, (0, 3, 3), [       # the recurrence only (no pages at all), all of it looped
    wkv(3, 10, 6, moe(12, 5, 2, 2.0, None, 20)),
    wkv(1, 70, 16, dense(30)),
    wkv(5, 4, 1, None),
])
UD = model(256, 128, 0.5, 1e-6, 20.0, (0, 2, 2), [    # sizes of the tensor-core kernels, a rank of 128, 16 heads
    wkv(2, 64, 32, moe(64, 8, 2, 1.5, (4, 1), 96)),
    lat(16, 32, 32, 16, 96, 128, 0.15, dense(160), (20000.0, 32, (8.0, 512, 16.0, 2.0))),
    wkv(4, 32, 8, moe(48, 16, 4, 3.0, (2, 1), 32)),
])
UE = model(77, 100, 1.3, 1e-5, 1.0, (2, 4, 2), [      # nothing a multiple of 8; the loop covers the last layers
    wkv(3, 14, 5, moe(20, 9, 2, 0.9, (3, 2), 10)),
    lat(3, 10, 6, 14, 22, 20, 0.35, moe(12, 7, 3, 1.2, None, 6), (5000.0, 6, (1.0, 128, 4.0, 4.0))),
    lat(7, 6, 2, 10, 30, 26, 0.4, None, (2.0, 2, (3.0, 6.5, 1.0, 0.01))),
    wkv(2, 130, 24, dense(36)),
])
UF = model(40, 32, 1.5, 1e-5, 3.0, (0, 1, 1), [wkv(2, 16, 4, dense(24))])
UG = model(48, 40, 1.0, 1e-4, 8.0, None, [lat(2, 12, 4, 20, 12, 12, 0.5, moe(16, 3, 3, 0.4, None, 8), (77.0, 4, (5.0, 30, 1.5, 1.0)))])
# name -> (config, seed, weight std, page size)
TINY = {"UA": (UA, 65, 0.16, 4), "UB": (UB, 52, 0.18, 8), "UC": (UC, 68, 0.18, 16), "UD": (UD, 64, 0.12, 16),
        "UE": (UE, 72, 0.1, 8), "UF": (UF, 56, 0.25, 8), "UG": (UG, 57, 0.25, 4)}


def arrange(name, t, gen):
    """The tensors that are drawn on their own (see the top of this file)."""
    draw = lambda: torch.rand(t.shape, generator=gen)
    if ".mu." in name:
        return draw()
    if name.endswith(".w0"):
        v = draw() * 2 - 1
        v[::2] -= 6.0
        return v
    if name.endswith("mix.u"):
        return draw() * 3 - 0.5
    if name.endswith(".router"):
        return t.float() * (6.0 / (float(t.float().std()) * t.shape[1] ** 0.5))
    if name.endswith(".correction"):
        # choice scores on both sides of zero, apart also where scores saturate
        return torch.randperm(t.shape[0], generator=gen) * (0.8 / t.shape[0]) - 1.1
    if name == "loop.step":
        return draw() * 2 - 1
    return t


def make_model_dir(root, name, dtype=torch.bfloat16):
    from rllm_b200.config import config_from_dict
    from rllm_b200.weights import write_random_model
    from rllm_b200.weights.random_init import random_tensors
    from rllm_b200.weights.safetensors_io import write_safetensors
    cfg, seed, std, _ = TINY[name]
    d = os.path.join(str(root), f"tiny_{name}_{str(dtype).split('.')[-1]}")
    if not os.path.isdir(d):
        write_random_model(cfg, seed, d, std=std, norm_std=0.3, dtype=dtype)
        arch, c = config_from_dict(cfg)
        gen = torch.Generator().manual_seed(seed + 1000)
        tensors = {n: arrange(n, t, gen).to(dtype).contiguous() for n, t in
                   random_tensors(arch.build(c), seed, std, 0.3, dtype).items()}
        write_safetensors(os.path.join(d, "model.safetensors"), tensors)
    return d


def random_prompt(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
