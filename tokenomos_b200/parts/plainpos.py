"""A position part that does nothing to q and k: positions do not enter the scores (order then comes
from elsewhere in the model: a recurrent layer, a causal mask's shape). It owns what every position part
owns, the step between the fused q/k/v projection and attention over the cache: the new keys and values
go into the paged pool and the queries come back as the attention kernels take them.

``maps`` > 1: a query head and a key head consist of that many parts, one per score map; map m of a head
reads part m of both. The part hands each map to the kernels as a head of its own, of the key's full
width with zeros outside its part, so that the kernels' ``q . k`` is the map's score against keys that are
stored once (``[T, heads, maps, dim] -> [T, heads * maps, maps * dim]``).

``head_norm``: an RMS norm over every q head and every k head (with the head layout's weights, or none), in the same
kernel as the write, which can also mix the values with another layer's (``encode_qk(..., mix=...)``).

``q_norm`` / ``k_norm``: an RMS norm over a token's whole query row and whole key row (all heads at once, before they
are split) with weights of those sizes, in the same kernel as the write.
"""

from __future__ import annotations

import torch

from tokenomos_b200 import ops
from tokenomos_b200.parts.contract import HeadLayout, StepContext, ValueRows
from tokenomos_b200.parts.registry import Runtime, register


class PlainQKV:
    capture_safe = True

    def __init__(self, maps: int = 1, q_norm: torch.Tensor | None = None, k_norm: torch.Tensor | None = None,
                 eps: float = 0.0, head_norm: bool = False):
        self.maps = int(maps)
        self.head_norm = self.takes_value_mix = bool(head_norm)
        if self.maps < 1:
            raise ValueError(f"plain q/k/v: {maps} maps")
        if self.maps > 1 and (q_norm is not None or head_norm):
            raise ValueError("plain q/k/v: norms over whole rows or heads go with one map a head")
        if head_norm and q_norm is not None:
            raise ValueError("plain q/k/v: norms over the whole rows or over the heads")
        self.q_norm = q_norm.float().reshape(-1).contiguous() if q_norm is not None else None
        self.k_norm = k_norm.float().reshape(-1).contiguous() if k_norm is not None else None
        self.eps = float(eps)

    def encode_qk(self, qkv, ctx: StepContext, heads: HeadLayout, pool, table, mix: ValueRows | None = None):
        if self.head_norm:
            if heads.v_is_k:
                raise ValueError("plain q/k/v: values that are the keys are not built here")
            return ops.qkv_head_norm_write(
                qkv, heads.q_norm, heads.k_norm, self.eps, ctx.positions, ctx.tok_seq, table, pool, heads.heads, heads.kv_heads,
                heads.head_dim, heads.v_dim or heads.head_dim, mix.rows if mix is not None else None,
                mix.lam if mix is not None else 0.0)
        if heads.q_norm is not None or heads.k_norm is not None or heads.v_is_k:
            raise ValueError("plain q/k/v: per-head norms and values that are the keys are not built here")
        if heads.heads % self.maps or heads.head_dim % self.maps:
            raise ValueError(f"plain q/k/v: {heads.heads} heads of {heads.head_dim} in {self.maps} maps")
        if self.q_norm is not None:
            return ops.qkv_row_norm_write(qkv, self.q_norm, self.k_norm, self.eps, ctx.positions, ctx.tok_seq, table, pool,
                                          heads.heads, heads.kv_heads, heads.head_dim, heads.v_dim or heads.head_dim)
        return ops.qkv_maps_write(qkv, ctx.positions, ctx.tok_seq, table, pool, heads.heads // self.maps,
                                  heads.kv_heads, heads.head_dim // self.maps, heads.v_dim or heads.head_dim, self.maps)


@register("position", "plain")
def build_plain_qkv(params: dict, tensors: dict, rt: Runtime) -> PlainQKV:
    return PlainQKV(params.get("maps", 1), tensors.get("q_norm"), tensors.get("k_norm"), params.get("eps", 0.0),
                    params.get("head_norm", False))
