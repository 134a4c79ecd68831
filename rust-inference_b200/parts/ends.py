"""The two ends of the model: token ids in, logits out.

``embedding``: h[t] = table[ids[t]] as float32 rows of the residual stream (times the record's
``scale``, 1 by default, and repeated ``copies`` times for a residual kept as several streams), passed through a
norm if the record names one; an id
outside the table is reported through the error word (thanhauco/rust-inference
src/ops/embedding.rs:10-42).

``linear`` head: logits = x W^T, no bias, float32 out of the float32 accumulator
(src/models/qwen3.rs:166-171, 286); a record may give a factor on the logits and a soft-cap
(cap * tanh(logits / cap)) applied after it.  When the model ties its embeddings the head is
given the embedding's table instead of a tensor of its own.

Another architecture registers other kinds (a scaled embedding, a head with a soft-cap or a bias)
with ``@register_embedding`` / ``@register_head`` and names them in its ``ModelSpec``.

Interfaces: embedding ``__call__(ids, ctx) -> float32 [tokens, hidden]`` (``ctx`` is the step's
:class:`~.base.StepContext`: an embedding that adds learned positions reads ``ctx.tok_pos``) and
``table`` (what a tied head shares); head ``__call__(x) -> float32 [rows, vocab]``, ``load(tensors)``
where ``tensors["weight"]`` is its own tensor or the embedding's table.
"""
from __future__ import annotations

import torch

from .. import ops
from .base import BuildEnv, CacheRequest, Part
from .registry import ParamInfo, build_part, part_class, register_embedding, register_head


@register_embedding("embedding")
class TokenEmbedding(Part):
    graph_safe = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.norm = None
        if getattr(spec, "norm", None) is not None:
            if getattr(spec, "copies", 1) != 1:
                raise ValueError("an embedding whose rows are normed has one stream")
            # the normed rows are the residual: float32 whatever the compute dtype
            self.norm = build_part("norm", spec.norm, BuildEnv(torch.float32, env.device))

    @classmethod
    def param_infos(cls, spec):
        infos = {"weight": ParamInfo((spec.vocab_size, spec.hidden_size), "matrix")}
        if getattr(spec, "norm", None) is not None:
            for local, info in part_class("norm", spec.norm).param_infos(spec.norm).items():
                infos["norm" + local] = info
        if getattr(spec, "side_width", 0):
            infos[spec.side_name] = ParamInfo((spec.vocab_size, spec.side_width), "matrix")
        return infos

    def load(self, tensors):
        self.table = tensors["weight"]
        if self.norm is not None:
            self.norm.load({k[len("norm"):]: v for k, v in tensors.items() if k.startswith("norm")})
        # a second table of token rows: the layers' token-fed sublayers read their columns of it
        self.side = tensors[self.spec.side_name] if getattr(self.spec, "side_width", 0) else None

    def weight_bytes(self):
        return self.table.numel() * self.table.element_size()

    def __call__(self, ids, ctx=None):
        if self.norm is not None:
            scale = getattr(self.spec, "scale", 1.0)
            if hasattr(self.norm, "of_rows"):
                return self.norm.of_rows(ids, self.table, scale)
            return self.norm(ops.embed(ids, self.table, scale))
        return ops.embed(ids, self.table, getattr(self.spec, "scale", 1.0), getattr(self.spec, "copies", 1))


@register_embedding("pair_hash")
class PairHashEmbedding(Part):
    """Token rows plus rows of a hashed table of (previous token, token) pairs; the previous token of a step's first
    token is per-sequence state (one int32 per cache slot), which the part asks the cache for."""
    graph_safe = True

    @classmethod
    def param_infos(cls, spec):
        return {"weight": ParamInfo((spec.vocab_size, spec.hidden_size), "matrix"),
                spec.pairs_name: ParamInfo((spec.buckets + 1, spec.hidden_size), "matrix")}

    def load(self, tensors):
        self.table = tensors["weight"]
        self.pairs = tensors[self.spec.pairs_name]

    def weight_bytes(self):
        return (self.table.numel() + self.pairs.numel()) * self.table.element_size()

    def cache_request(self):
        return CacheRequest(state_shape=(1,), state_dtype=torch.int32)

    def __call__(self, ids, ctx, cache):
        s = self.spec
        return ops.embed_pair_hash(ids, self.table, self.pairs, cache.state.view(-1), ctx.tok_seq, ctx.tok_pos, ctx.seq_slot,
                                   ctx.seq_start, s.mul_prev, s.mul_cur, single=ctx.decode_only)


@register_head("linear")
class LinearHead(Part):
    graph_safe = True

    @classmethod
    def param_infos(cls, spec):
        return {"weight": ParamInfo((spec.vocab_size, spec.hidden_size), "matrix")}

    def load(self, tensors):
        self.weight = tensors["weight"]

    def weight_bytes(self):
        return self.weight.numel() * self.weight.element_size()

    def reads_first(self):
        return self.weight

    def __call__(self, x):
        z = ops.scale_(ops.linear(x, self.weight, out_dtype=torch.float32), getattr(self.spec, "scale", 1.0))
        return ops.softcap_(z, getattr(self.spec, "softcap", 0.0))
