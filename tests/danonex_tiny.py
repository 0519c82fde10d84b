"""The tests' own small Danonex configurations and model folders. They differ from each other in every size and option:
heads that share keys and heads that do not, key and value sizes that differ (and that are equal), a rotation of a part
of a head, of all of it and none, with the yarn rule (ramps inside the head, cut off at either end, of no width) and
without, bounds that bite and bounds that hardly do and none, convolutions of one tap to five, delta-rule heads narrower
than a warp and wider, factors of 1 and other numbers, layers without a feed-forward, models of one kind of layer, and of
one layer."""
import os

import torch


def delta(heads, kv_heads, dim, vdim, conv, ff):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": dense(ff)}


def att(heads, kv_heads, dim, vdim, scale, ff, softcap=None, rot=None):
    """rot: (base, dims, None or (factor, original, fast, slow))"""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if rot[2] is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    return {"type": "attention", "mixer": m, "mlp": dense(ff)}


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def model(vocab, width, eps, mult, logit_scale, layers):
    return {"architecture": "Danonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "logit_scale": logit_scale, "layers": layers}


DA = model(130, 72, 1e-5, 0.7, 1.5, [      # both kinds, every option; a bound that bites; a ramp inside the head
    att(4, 2, 24, 40, 0.4, 96, 3.0, (800.0, 16, (4.0, 64, 8.0, 1.0))),
    delta(4, 2, 24, 16, 4, None),
    att(3, 3, 16, 24, 0.5, None, 20.0, (100.0, 16, (2.5, 100, 3.0, 0.5))),
    delta(2, 2, 40, 24, 2, 56),
])
DB = model(200, 60, 3e-6, 1.0, 1.0, [      # attention only; no bound, no rotation, a rotation without scaling
    att(5, 1, 12, 12, 0.3, 44),
    att(2, 2, 20, 8, 0.25, None, None, (10000.0, 8, None)),
    att(6, 3, 8, 32, 0.6, 40, 1.25, (50.0, 8, (16.0, 4096, 32.0, 1.0))),
])
DC = model(90, 52, 1e-6, 0.25, 3.0, [      # the delta rule only: nothing is paged; one tap, heads of few channels, wide heads
    delta(3, 1, 10, 14, 1, 30),
    delta(6, 3, 5, 6, 5, None),
    delta(1, 1, 70, 9, 3, 24),
    delta(2, 1, 8, 130, 2, None),
])
DD = model(256, 128, 1e-6, 0.6, 0.5, [     # equal head sizes of 64 and 128, compiled scan sizes, pages of 16
    att(8, 2, 64, 64, 0.2, 160, 12.0, (20000.0, 32, (8.0, 512, 16.0, 2.0))),
    delta(4, 2, 64, 64, 4, 128),
    att(2, 1, 128, 128, 0.12, 96, 30.0, (500.0, 128, (3.0, 2048, 64.0, 1.0))),
    delta(2, 1, 128, 32, 3, None),
    att(2, 2, 64, 64, 0.1, None, None, (1e6, 64, None)),
])
DE = model(160, 96, 1e-5, 1.5, 2.5, [      # unequal head sizes in steps of 16 (mma.sync), many heads a key
    att(16, 2, 32, 48, 0.35, 64, 5.0, (300.0, 20, (2.0, 40, 2.0, 1.0))),
    att(4, 4, 80, 16, 0.15, 72, 8.0, (5000.0, 80, (1.0, 128, 4.0, 4.0))),
    delta(8, 4, 32, 24, 3, 88),
])
DF = model(40, 32, 1e-5, 0.5, 4.0, [delta(1, 1, 16, 16, 3, 24)])
DG = model(48, 40, 1e-4, 2.0, 1.0, [att(1, 1, 20, 12, 0.5, 16, 2.0, (77.0, 6, (5.0, 30, 1.5, 1.0)))])
# name -> (config, seed, weight std, page size)
TINY = {"DA": (DA, 41, 0.15, 4), "DB": (DB, 42, 0.16, 8), "DC": (DC, 43, 0.18, 16), "DD": (DD, 44, 0.1, 16),
        "DE": (DE, 45, 0.12, 16), "DF": (DF, 46, 0.25, 8), "DG": (DG, 47, 0.25, 4)}


def make_model_dir(root, name, dtype=torch.bfloat16):
    from rllm_b200.weights import write_random_model
    cfg, seed, std, _ = TINY[name]
    d = os.path.join(str(root), f"tiny_{name}_{str(dtype).split('.')[-1]}")
    if not os.path.isdir(d):
        write_random_model(cfg, seed, d, std=std, norm_std=0.3, dtype=dtype)
    return d


def random_prompt(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
