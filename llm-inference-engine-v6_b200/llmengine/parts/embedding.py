"""Token embedding and output head.

"lookup": the residual stream starts as the table row of each token id, widened to float32
(embed_lookup_f32, src/kernels.cpp:59-66). "linear": logits = x . W^T without bias for the rows
whose logits are wanted (src/engine.cpp:415-433); with tied embeddings W is the embedding table
itself (src/model.cpp:184-195). Variants (a scaled embedding, a capped or biased head) are other
registered kinds; the model only knows the two interfaces.
"""
from __future__ import annotations

from typing import List

import torch

from .base import Embedding, Head, NormalizedRows, StateNeed
from .registry import build_part, part_class, register_part
from .spec import EmbeddingSpec, HeadSpec, TensorNeed


class TokenLookup(Embedding):
    def __init__(self, spec: EmbeddingSpec, env):
        super().__init__(spec, env)
        self.table = None

    @staticmethod
    def tensor_needs(spec: EmbeddingSpec) -> List[TensorNeed]:
        return [TensorNeed(spec.weight, (spec.vocab_size, spec.dim), "compute")]

    def load(self, tensors) -> None:
        self.table = tensors[self.spec.weight]

    def forward(self, ctx) -> torch.Tensor:
        ops, n = self.env.ops, ctx.n_tokens
        h = ctx.ws.get("model.residual", (n, self.spec.dim), torch.float32)
        scale = float(getattr(self.spec, "scale", 1.0))
        if scale != 1.0:
            return ops.embed(self.table, ctx.token_ids, h, scale=scale)
        nxt = getattr(ctx, "next_norm", None)
        wn = nxt.prescale_weight() if nxt is not None else None
        if (self.env.dtype == torch.bfloat16 and getattr(ops, "meet_products", False) and n <= 64 and wn is not None and
                wn.numel() == self.spec.dim and wn.dtype == torch.float32):
            # a step of few tokens: the gather has the rows in its hands, so it leaves what the first norm
            # needs beside them (its weight times the rows, and the rows' sums of squares), and that norm
            # is no kernel of its own
            ctx.stream_sumsq = ctx.ws.get("embedding.sumsq", (n, 1), torch.float32)
            scaled = ctx.ws.get("stream.prescaled", (n, self.spec.dim), torch.bfloat16)
            ctx.stream_prescaled = (scaled, wn)
            return ops.embed(self.table, ctx.token_ids, h, sumsq=ctx.stream_sumsq, next_w=wn, scaled=scaled)
        if self.env.dtype == torch.bfloat16 and hasattr(ops, "few_token_splits") and ops.few_token_splits(128, self.spec.dim, n, "plain") > 0:
            # a step of few tokens: the first norm can be folded into the product after it if the
            # rows' sums of squares are known; the gather has the rows in its hands anyway
            ctx.stream_sumsq = ctx.ws.get("embedding.sumsq", (n, 1), torch.float32)
            return ops.embed(self.table, ctx.token_ids, h, sumsq=ctx.stream_sumsq)
        return ops.embed(self.table, ctx.token_ids, h)


    def lookup(self, ctx, out: torch.Tensor) -> torch.Tensor:
        scale = float(getattr(self.spec, "scale", 1.0))
        return self.env.ops.embed(self.table, ctx.token_ids, out, **({} if scale == 1.0 else {"scale": scale}))


class NormedTokenLookup(TokenLookup):
    """The table row of each token id, then a norm of its own over the row: the float32 stream starts normalised. The norm is any
    registered norm (EmbeddingSpec.norm); it reads the gathered rows and writes the stream in float32."""

    def __init__(self, spec: EmbeddingSpec, env):
        super().__init__(spec, env)
        if spec.norm is None:
            raise ValueError("embedding 'lookup_normed' needs a norm")
        self.norm = build_part("norm", spec.norm, env)

    @staticmethod
    def tensor_needs(spec: EmbeddingSpec) -> List[TensorNeed]:
        return TokenLookup.tensor_needs(spec) + list(part_class("norm", spec.norm.kind).tensor_needs(spec.norm))

    def subparts(self):
        return (self.norm,)

    def load(self, tensors) -> None:
        super().load(tensors)
        self.norm.load(tensors)

    def forward(self, ctx) -> torch.Tensor:
        return self.lookup(ctx, ctx.ws.get("model.residual", (ctx.n_tokens, self.spec.dim), torch.float32))

    def lookup(self, ctx, out: torch.Tensor) -> torch.Tensor:
        raw = ctx.ws.get("embedding.rows", (ctx.n_tokens, self.spec.dim), torch.float32)
        super().lookup(ctx, raw)
        return self.norm.run(raw, ctx, None, ctx.n_tokens, out=out)


class PairLookup(TokenLookup):
    """The table row of each token id times `scale`, plus a row of a second table chosen by the token and the one before it
    (EmbeddingSpec "lookup_pairs"). One kernel: a portion's first token finds its predecessor in the request's slot, which afterwards
    holds the portion's last token; position 0 has none and takes the row behind the buckets."""

    def __init__(self, spec: EmbeddingSpec, env):
        super().__init__(spec, env)
        if not spec.pair_weight or spec.pair_buckets < 1 or min(spec.pair_mul_prev, spec.pair_mul_cur) < 0:
            raise ValueError("embedding 'lookup_pairs' needs the pair table, at least one bucket and multipliers that are not negative")
        self.pairs = None

    @staticmethod
    def tensor_needs(spec: EmbeddingSpec) -> List[TensorNeed]:
        return TokenLookup.tensor_needs(spec) + [TensorNeed(spec.pair_weight, (spec.pair_buckets + 1, spec.dim), "compute")]

    def cache_needs(self):
        return (StateNeed("embedding.previous", (1,), torch.int32),)

    def load(self, tensors) -> None:
        super().load(tensors)
        self.pairs = tensors[self.spec.pair_weight]

    def forward(self, ctx) -> torch.Tensor:
        s = self.spec
        h = ctx.ws.get("model.residual", (ctx.n_tokens, s.dim), torch.float32)
        return self.env.ops.embed_pairs(self.table, self.pairs, s.pair_buckets, s.pair_mul_prev, s.pair_mul_cur, float(s.scale),
                                        ctx.embedding_cache.states["embedding.previous"], ctx, h)

    def lookup(self, ctx, out: torch.Tensor) -> torch.Tensor:
        # the slot has moved on to the portion's last token: the rows are taken from the stream, which nobody has written yet
        return out.copy_(ctx.ws.get("model.residual", (ctx.n_tokens, self.spec.dim), torch.float32))


class LinearHead(Head):
    def __init__(self, spec: HeadSpec, env):
        super().__init__(spec, env)
        self.weight = None

    @staticmethod
    def tensor_needs(spec: HeadSpec) -> List[TensorNeed]:
        return [TensorNeed(spec.weight, (spec.vocab_size, spec.dim), "compute")]

    def load(self, tensors) -> None:
        self.weight = tensors[self.spec.weight]

    def wants_lazy_norm(self, ctx) -> bool:
        # every request of the step brings one token and wants its logits: the wanted rows are all rows, in order
        return (self.env.dtype == torch.bfloat16 and getattr(self.env.ops, "meet_products", False) and
                0 < ctx.n_rows == ctx.n_tokens == ctx.n_seqs <= 64)

    def forward(self, x, ctx) -> torch.Tensor:
        n = x.n if isinstance(x, NormalizedRows) else x.shape[0]
        logits = ctx.ws.get("model.logits", (max(n, 1), self.spec.vocab_size), torch.float32)[:n]
        cap = float(getattr(self.spec, "softcap", 0.0) or 0.0)
        done = False
        if isinstance(x, NormalizedRows):
            ops = self.env.ops
            if x.prescaled is not None and n and self.wants_lazy_norm(ctx) and ops.can_meet(x.prescaled[:n], self.weight):
                # the product runs on weight * rows and divides by the rows' root mean square in its epilogue
                ops.gemm_scaled(x.prescaled[:n], self.weight, logits, x.row_scale(ops))
                done = True
            else:
                x = x.dense(ctx)
        if n and not done:
            self.env.ops.gemm(x, self.weight, logits)
        if n and cap > 0.0:
            self.env.ops.softcap(logits, cap)  # logits <- cap * tanh(logits / cap), float32
        return logits


register_part("embedding", "lookup", TokenLookup)
register_part("embedding", "lookup_normed", NormedTokenLookup)
register_part("embedding", "lookup_pairs", PairLookup)
register_part("head", "linear", LinearHead)
