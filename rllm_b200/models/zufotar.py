"""Zufotar assembled from parts: layers whose mixer and feed-forward run side by side, each behind a norm of its own
(`ParallelBlock` with two norms). The mixer is attention over compressed latents with a latent in front of the queries, a
rotated part with scaled frequencies and an output gate per number (pages of latents), or a recurrence with a bonus behind
a token shift (`TimeMixing`, a state); the feed-forward is dense with the erf form of gelu, a mixture of gated experts
with a gated shared expert, or absent. A stretch of layers may run several times with the same weights: every run has a
cache layer of its own, every pass begins with a learned vector, all but the first also with the embedding's output
again. Tensor names: `embed`, `loop.step`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`; the output
matrix is the embedding table, the logits are bounded. Everything numeric that can differ between models comes from the
configuration."""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.zufotar import ZufotarConfig
from ..parts import (ActFFN, Embedding, GluFFN, GluRoutedExperts, InterleavedRotary, LatentAttention, LoopStep, ParallelBlock,
                     RMSNorm, TimeMixing, make_part)
from .model import Model, looped_schedule

SUM_EPS = 1e-20           # added to the sum that the chosen experts' scores are divided by


def _mixer(cfg: ZufotarConfig, layer):
    m, W, eps = layer.mixer, cfg.width, cfg.norm_eps
    if layer.type == "latent_attention":
        position = InterleavedRotary(m.rot_dim, m.rot_base, m.rot_dims, m.rot_scaling) if m.rot_dim else None
        return LatentAttention(W, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, position, eps=eps, gate="full",
                               q_rank=m.q_rank)
    if layer.type == "wkv":
        return TimeMixing(W, m.heads, m.dim, eps=eps, decay_rank=m.decay_rank)
    raise ValueError(f"no mixer for layer type {layer.type!r}")


def _ffn(cfg: ZufotarConfig, f):
    if f.kind == "dense":
        return ActFFN(cfg.width, f.ff, "gelu_erf")
    shared = None if f.shared_ff is None else GluFFN(cfg.width, f.shared_ff, "silu")
    return GluRoutedExperts(cfg.width, f.ff, f.experts, f.top, "silu", score="sigmoid", renorm=True, shared=shared,
                            shared_gate=True, correction=True, groups=f.groups, keep=f.keep, group_sum=2, sum_eps=SUM_EPS,
                            weight_scale=f.scale)


def build_zufotar(cfg: ZufotarConfig) -> Model:
    W, eps = cfg.width, cfg.norm_eps
    emb = Embedding(cfg.vocab, W, name="embed", scale=cfg.embedding_scale)
    emb.prefix = ""
    blocks, steps = [], []
    for i, layer in enumerate(cfg.layers):
        ffn = None if layer.mlp is None else _ffn(cfg, layer.mlp)
        block = ParallelBlock(RMSNorm(W, eps, "norm1"), _mixer(cfg, layer), ffn,
                              ffn_norm=None if ffn is None else RMSNorm(W, eps, "norm2"))
        block.set_prefix(f"l{i}.")
        blocks.append(block)
    for t in range(cfg.loop_times if cfg.has_loop else 0):
        step = LoopStep(W, cfg.loop_times, t, owner=steps[0] if steps else None, embedding=emb if t else None)
        step.prefix = "loop."
        steps.append(step)
    schedule = looped_schedule(blocks, cfg.layer_runs(), steps)
    final_norm = RMSNorm(W, eps, "norm")
    final_norm.prefix = "final."
    head = make_part("head", "linear", vocab=cfg.vocab, hidden=W, norm=final_norm, tied_to=emb, softcap=cfg.logit_softcap)
    head.prefix = ""
    model = Model(cfg, emb, blocks, schedule, head, prefix="")
    # a layer without feed-forward has no use for the norm in front of one, should a checkpoint carry it
    model.ignorable = tuple(f"l{i}.norm2" for i, layer in enumerate(cfg.layers) if layer.mlp is None)
    return model


register_architecture("Zufotar", ZufotarConfig, build_zufotar, model_types=("zufotar",))
