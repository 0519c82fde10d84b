"""Danonex assembled from parts: layers that norm a sublayer's output on its way into the stream (`OutputNormBlock`), whose
mixer is the gated delta rule with one decay per head (a state) or grouped-query attention with queries and keys normed
over all heads together, an interleaved rotation with scaled frequencies, bounded scores and a sink (pages); the
feed-forward is dense with the erf form of gelu, or absent. The factor on the logits is folded into the final norm. Tensor
names: `embed`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`, `l<i>.mlp.{up,down}`, `final.norm`; the output matrix is the
embedding table. Everything numeric that can differ between models comes from the configuration."""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.danonex import DanonexConfig
from ..parts import ActFFN, DeltaRuleMixer, Embedding, InterleavedRotary, OutputNormBlock, RMSNorm, SinkGQAttention, make_part
from .model import LayerCall, Model

UNIT_EPS = 1e-6           # under the root of the delta rule's unit vectors


def _mixer(cfg: DanonexConfig, layer):
    m, W, eps = layer.mixer, cfg.width, cfg.norm_eps
    if layer.type == "delta":
        return DeltaRuleMixer(W, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, eps, UNIT_EPS, decay="head", gate="full")
    if layer.type == "attention":
        position = InterleavedRotary(m.dim, m.rot_base, m.rot_dims, m.rot_scaling) if m.rot_dims else None
        return SinkGQAttention(W, m.heads, m.kv_heads, m.dim, m.vdim, position=position, scale=m.scale, qk_norm=True,
                               qk_norm_span="row", sink=True, softcap=m.softcap, eps=eps)
    raise ValueError(f"no mixer for layer type {layer.type!r}")


def build_danonex(cfg: DanonexConfig) -> Model:
    W, eps = cfg.width, cfg.norm_eps
    emb = Embedding(cfg.vocab, W, name="embed")
    emb.prefix = ""
    blocks = []
    for i, layer in enumerate(cfg.layers):
        ffn = None if layer.ff is None else ActFFN(W, layer.ff, "gelu_erf")
        block = OutputNormBlock(_mixer(cfg, layer), RMSNorm(W, eps, "norm1"), ffn,
                                None if ffn is None else RMSNorm(W, eps, "norm2"), coef=cfg.residual_mult)
        block.set_prefix(f"l{i}.")
        blocks.append(block)
    schedule = [LayerCall(i, i, True) for i in range(len(blocks))]
    final_norm = RMSNorm(W, eps, "norm", scale=cfg.logit_scale)
    final_norm.prefix = "final."
    head = make_part("head", "linear", vocab=cfg.vocab, hidden=W, norm=final_norm, tied_to=emb)
    head.prefix = ""
    return Model(cfg, emb, blocks, schedule, head, prefix="")


register_architecture("Danonex", DanonexConfig, build_danonex, model_types=("danonex",))
