"""How a layer's parts are arranged. Pre-norm residual block, the reference's Llama layer
order (src/model/registry/llama.rs:163-245): h += mixer(norm(h)); h += ffn(norm(h)).
`SandwichBlock` norms each sublayer's output as well: h += norm_b(mixer(norm(h))), the same for
the feed-forward, which may be absent. `LoopStep` is a block that only adds a learned vector to
every row, and before it the embedding's output again where it is given the embedding: what a pass of a looped stretch of
layers begins with. `PostNormBlock` norms after the sum,
h = norm(alpha h + sublayer(h)), the sublayers reading the stream itself; `OutputNormBlock` norms the sublayer's output
alone, h += coef * norm(sublayer(h)), the sublayers again reading the stream itself. `ParallelBlock` has one norm whose
output both sublayers read, or one norm each: h += mixer(n) + ffn(n), n = norm(h), or
h += mixer(norm1(h)) + ffn(norm2(h)). `GatedPreNormBlock` is the pre-norm order with a
gate on each sublayer's way into the stream: h += sigmoid(W_g n + b_g) * sublayer(n), n = norm(h), W_g a square matrix."""
from __future__ import annotations

from .base import Param, Part, Source, register_part


class PreNormBlock(Part):
    """`names` maps the four parts to their checkpoint sub-prefixes."""
    graph_safe = True

    def __init__(self, mixer_norm: Part, mixer: Part, ffn_norm: Part, ffn: Part,
                 names=("input_layernorm.", "self_attn.", "post_attention_layernorm.", "mlp.")):
        self.mixer_norm, self.mixer, self.ffn_norm, self.ffn = mixer_norm, mixer, ffn_norm, ffn
        self.names = names

    def children(self):
        return [self.mixer_norm, self.mixer, self.ffn_norm, self.ffn]

    def set_prefix(self, prefix: str):
        self.prefix = prefix
        for part, sub in zip(self.children(), self.names):
            part.prefix = prefix + sub
            for c in part.children():
                if not c.prefix:
                    c.prefix = part.prefix

    def cache_spec(self):
        return self.mixer.cache_spec()

    def forward(self, h, ctx, cache):
        """h: float32 residual stream [T, hidden], updated in place."""
        self.mixer.forward(self._norm(self.mixer_norm, self.mixer, h, ctx), ctx, cache, h)
        self.ffn.forward(self._norm(self.ffn_norm, self.ffn, h, ctx), ctx, h)
        return h

    @staticmethod
    def _norm(norm, consumer, h, ctx):
        """A consumer that hands its input straight to the backend's products (`takes_deferred`)
        gets the norm in deferred form, so that it can run inside the first product."""
        if getattr(consumer, "takes_deferred", False) and hasattr(norm, "deferred"):
            return norm.deferred(h, ctx)
        return norm.forward(h, ctx)


class SandwichBlock(Part):
    """A norm before and after each sublayer. The post-norm, the sum over a routed feed-forward's
    parts and the residual sum are one float kernel. `names`: checkpoint sub-prefixes of mixer and
    feed-forward; the four norms' weights are tensors named `norm_names` under the block's prefix."""
    graph_safe = True

    def __init__(self, mixer_norm: Part, mixer: Part, mixer_post: Part, ffn_norm: Part | None = None,
                 ffn: Part | None = None, ffn_post: Part | None = None, names=("mix.", "mlp.")):
        self.mixer_norm, self.mixer, self.mixer_post = mixer_norm, mixer, mixer_post
        self.ffn_norm, self.ffn, self.ffn_post = ffn_norm, ffn, ffn_post
        self.names = names

    def children(self):
        return [p for p in (self.mixer_norm, self.mixer, self.mixer_post, self.ffn_norm, self.ffn, self.ffn_post)
                if p is not None]

    def set_prefix(self, prefix: str):
        self.prefix = prefix
        for norm in (self.mixer_norm, self.mixer_post, self.ffn_norm, self.ffn_post):
            if norm is not None:
                norm.prefix = prefix            # a norm's tensor is named by its `weight_name`
        for part, sub in ((self.mixer, self.names[0]), (self.ffn, self.names[1])):
            if part is not None:
                part.prefix = prefix + sub
                for c in part.children():
                    if not c.prefix:
                        c.prefix = part.prefix

    def cache_spec(self):
        return self.mixer.cache_spec()

    def forward(self, h, ctx, cache):
        """h: float32 residual stream [T, hidden], updated in place."""
        be = ctx.backend
        x = PreNormBlock._norm(self.mixer_norm, self.mixer, h, ctx)
        be.rmsnorm_add(h, self._output(self.mixer, h, x, ctx, cache), self.mixer_post.weight_f32(), self.mixer_post.eps)
        if self.ffn is not None:
            x = PreNormBlock._norm(self.ffn_norm, self.ffn, h, ctx)
            be.rmsnorm_add(h, self._output(self.ffn, h, x, ctx), self.ffn_post.weight_f32(), self.ffn_post.eps)
        return h

    @staticmethod
    def _output(part, h, x, ctx, *cache):
        """The sublayer's float output: returned by parts that can (`returns_output`), else gathered
        in a zeroed buffer that stands in for the residual stream."""
        if getattr(part, "returns_output", False):
            return part.forward(x, ctx, *cache, None)
        import torch
        y = torch.zeros_like(h)
        part.forward(x, ctx, *cache, y)
        return y


class PostNormBlock(Part):
    """h <- norm1(alpha h + mixer(h)); h <- norm2(alpha h + ffn(h)) (the feed-forward may be absent). The
    sublayers read the stream itself, in the run's storage type; sum and norm are one float kernel, which
    also writes the copy that the next sublayer's products read. A feed-forward may return its output as
    `Summands` (parts to be added in order, and a second summand with a sigmoid gate per row), which that
    kernel takes as they come. `names`: checkpoint sub-prefixes of mixer and feed-forward; the norms'
    weights are tensors named by each norm's `weight_name` under the block's prefix."""
    graph_safe = True

    def __init__(self, mixer: Part, mixer_norm: Part, ffn: Part | None = None, ffn_norm: Part | None = None,
                 alpha: float = 1.0, names=("mix.", "mlp.")):
        self.mixer, self.mixer_norm, self.ffn, self.ffn_norm = mixer, mixer_norm, ffn, ffn_norm
        self.alpha, self.names = float(alpha), names

    def children(self):
        return [p for p in (self.mixer, self.mixer_norm, self.ffn, self.ffn_norm) if p is not None]

    def set_prefix(self, prefix: str):
        self.prefix = prefix
        for norm in (self.mixer_norm, self.ffn_norm):
            if norm is not None:
                norm.prefix = prefix
        for part, sub in ((self.mixer, self.names[0]), (self.ffn, self.names[1])):
            if part is not None:
                if hasattr(part, "set_prefix"):
                    part.set_prefix(prefix + sub)          # a part with named children of its own
                    continue
                part.prefix = prefix + sub
                for c in part.children():
                    if not c.prefix:
                        c.prefix = part.prefix

    def cache_spec(self):
        return self.mixer.cache_spec()

    @staticmethod
    def _finish(be, h, y, alpha, norm):
        return be.postnorm(h, y, alpha, norm.weight_f32(), norm.eps)

    def forward(self, h, ctx, cache):
        """h: float32 residual stream [T, hidden], updated in place."""
        be = ctx.backend
        kept = ctx.per_forward.get("stream_copy")
        x = kept[1] if kept is not None and kept[0] is h else be.stream_copy(h)
        y = self.mixer.forward(x, ctx, cache, None)
        x = self._finish(be, h, y, self.alpha, self.mixer_norm)
        if self.ffn is not None:
            y = self.ffn.forward(x, ctx, None)
            x = self._finish(be, h, y, self.alpha, self.ffn_norm)
        ctx.per_forward["stream_copy"] = (h, x)        # what the next block's mixer reads
        return h


class OutputNormBlock(PostNormBlock):
    """h += coef * norm1(mixer(h)); h += coef * norm2(ffn(h)) (the feed-forward may be absent). As in `PostNormBlock` the
    sublayers read the stream itself in the run's storage type; norm, coefficient and sum are one float kernel, which
    also writes the copy that the next sublayer's products read."""
    graph_safe = True

    def __init__(self, mixer: Part, mixer_norm: Part, ffn: Part | None = None, ffn_norm: Part | None = None,
                 coef: float = 1.0, names=("mix.", "mlp.")):
        super().__init__(mixer, mixer_norm, ffn, ffn_norm, alpha=coef, names=names)

    @staticmethod
    def _finish(be, h, y, coef, norm):
        return be.output_norm(h, y, coef, norm.weight_f32(), norm.eps)


class ParallelBlock(Part):
    """h <- h + (mixer(n) + ffn(n)) with n = norm(h): one norm, both sublayers read its output, the feed-forward may
    be absent. With `ffn_norm` the feed-forward reads a norm of its own of the same h; the two are made in one pass where
    they are not part of a product's kernel, and a mixer that norms the stream itself (`norms_stream`) makes both.
    Sublayers return their float outputs (a tensor, `Summands`, or `NormedSum` for a mixer whose members are
    normed before they are added); the sum of all of them and the residual sum are one float kernel. A mixer made
    of several mixers gets a tuple of cache layers. `names`: checkpoint sub-prefixes of mixer and feed-forward; the
    norm's weight is a tensor named by its `weight_name` under the block's prefix."""
    graph_safe = True

    def __init__(self, norm: Part, mixer: Part, ffn: Part | None = None, names=("mix.", "mlp."), ffn_norm: Part | None = None):
        self.norm, self.mixer, self.ffn, self.names, self.ffn_norm = norm, mixer, ffn, names, ffn_norm
        if getattr(mixer, "norms_stream", False) and ffn is not None and ffn_norm is None:
            raise ValueError("a mixer that norms the stream itself leaves no normed rows for the feed-forward")

    def children(self):
        return [p for p in (self.norm, self.ffn_norm, self.mixer, self.ffn) if p is not None]

    def set_prefix(self, prefix: str):
        self.prefix = prefix
        self.norm.prefix = prefix
        if self.ffn_norm is not None:
            self.ffn_norm.prefix = prefix
        for part, sub in ((self.mixer, self.names[0]), (self.ffn, self.names[1])):
            if part is None:
                continue
            if hasattr(part, "set_prefix"):
                part.set_prefix(prefix + sub)
                continue
            part.prefix = prefix + sub
            for c in part.children():
                if not c.prefix:
                    c.prefix = part.prefix

    def cache_spec(self):
        return self.mixer.cache_spec()

    def forward(self, h, ctx, cache):
        """h: float32 residual stream [T, hidden], updated in place."""
        be = ctx.backend
        if self.ffn_norm is None and not getattr(self.mixer, "norms_stream", False):
            n = n2 = self.norm.forward(h, ctx)
            m = self.mixer.forward(n, ctx, cache, None)
        else:
            # which norms run inside the first product of their sublayer
            inside = lambda part: part is not None and getattr(part, "takes_deferred", False) and be.fuses_norm(h.shape[0])
            n2 = self.ffn_norm.deferred(h, ctx) if inside(self.ffn) else None
            second = (self.ffn_norm.weight_f32(), self.ffn_norm.eps) if self.ffn is not None and n2 is None else None
            if getattr(self.mixer, "norms_stream", False):
                m, made = self.mixer.forward_stream(h, self.norm, ctx, cache, second)
                n2 = made if second is not None else n2
            elif second is not None and not inside(self.mixer):
                n, n2 = be.norm_pair(h, self.norm.weight_f32(), self.norm.eps, *second)
                m = self.mixer.forward(n, ctx, cache, None)
            else:
                n2 = self.ffn_norm.forward(h, ctx) if second is not None else n2
                m = self.mixer.forward(PreNormBlock._norm(self.norm, self.mixer, h, ctx), ctx, cache, None)
        f = None if self.ffn is None else self.ffn.forward(n2, ctx, None)
        return be.combine(h, m, f)


class GatedPreNormBlock(Part):
    """n = norm1(h); h += sigmoid(W_1 n + b_1) * mixer(n); then the same with norm2, W_2, b_2 and the feed-forward, which
    may be absent. The gates are as wide as the stream. A sublayer returns its float output (a tensor, or `ScaledSum`
    for a mixer made of mixers); the gate's sigmoid, the product with the output and the residual sum are one float
    kernel. `names`: checkpoint sub-prefixes of mixer and feed-forward; `gate_names`: the gates' matrices under the
    block's prefix (their biases: the same names with `.b`); the norms' weights are tensors named by each norm's
    `weight_name` under the block's prefix."""
    graph_safe = True

    def __init__(self, hidden: int, mixer_norm: Part, mixer: Part, ffn_norm: Part | None = None, ffn: Part | None = None,
                 names=("mix.", "mlp."), gate_names=("rg1", "rg2")):
        self.hidden, self.mixer_norm, self.mixer, self.ffn_norm, self.ffn = hidden, mixer_norm, mixer, ffn_norm, ffn
        self.names, self.gate_names = names, gate_names
        self.w_g1 = self.b_g1 = self.w_g2 = self.b_g2 = None

    def children(self):
        return [p for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if p is not None]

    def params(self):
        W = self.hidden
        g1, g2 = self.gate_names
        ps = [Param("w_g1", (Source(g1, (W, W)),)), Param("b_g1", (Source(g1 + ".b", (W,)),), role="vector")]
        if self.ffn is not None:
            ps += [Param("w_g2", (Source(g2, (W, W)),)), Param("b_g2", (Source(g2 + ".b", (W,)),), role="vector")]
        return ps

    def set_prefix(self, prefix: str):
        self.prefix = prefix
        for norm in (self.mixer_norm, self.ffn_norm):
            if norm is not None:
                norm.prefix = prefix
        for part, sub in ((self.mixer, self.names[0]), (self.ffn, self.names[1])):
            if part is None:
                continue
            if hasattr(part, "set_prefix"):
                part.set_prefix(prefix + sub)
                continue
            part.prefix = prefix + sub
            for c in part.children():
                if not c.prefix:
                    c.prefix = part.prefix

    def cache_spec(self):
        return self.mixer.cache_spec()

    def finalize(self, device, dtype):
        self._b1 = self.b_g1.float().contiguous()
        self._b2 = None if self.b_g2 is None else self.b_g2.float().contiguous()

    def forward(self, h, ctx, cache):
        """h: float32 residual stream [T, hidden], updated in place."""
        be = ctx.backend
        n = self.mixer_norm.deferred(h, ctx)
        gate = be.linear_f32(n, self.w_g1, tag="gate")
        be.gated_add(h, gate, self._b1, self.mixer.forward(n, ctx, cache, None))
        if self.ffn is not None:
            n = self.ffn_norm.deferred(h, ctx)
            gate = be.linear_f32(n, self.w_g2, tag="gate")
            be.gated_add(h, gate, self._b2, self.ffn.forward(n, ctx, None))
        return h


class LoopStep(Part):
    """h += table[index] on every row. The passes of one loop share the table [times, hidden]: the
    first owns the tensor (`owner` None), the others name the first. `embedding`: its output for the step's tokens is added
    first (looked up again, not kept)."""
    graph_safe = True

    def __init__(self, hidden: int, times: int, index: int, owner: "LoopStep | None" = None, name: str = "step",
                 embedding: Part | None = None):
        self.hidden, self.times, self.index, self.owner, self.name = hidden, times, index, owner, name
        self.embedding = embedding
        self.table = None

    def params(self):
        if self.owner is not None:
            return []
        return [Param("table", (Source(self.name, (self.times, self.hidden)),), role="vector")]

    def cache_spec(self):
        return None

    def finalize(self, device, dtype):
        table = (self.owner or self).table
        self._row = table[self.index].float().contiguous()

    def forward(self, h, ctx, cache=None):
        if self.embedding is None:
            return ctx.backend.add_row(h, self._row)
        return ctx.backend.add_row(h, self._row, ctx.token_ids, self.embedding.table, self.embedding.scale)


register_part("block", "prenorm", PreNormBlock)
register_part("block", "sandwich", SandwichBlock)
register_part("block", "postnorm", PostNormBlock)
register_part("block", "output_norm", OutputNormBlock)
register_part("block", "parallel", ParallelBlock)
register_part("block", "prenorm_gated", GatedPreNormBlock)
register_part("block", "loop_step", LoopStep)
