"""Mixer `gqa_attention`: grouped-query attention over the paged cache.

q = Wq h, k = Wk h, v = Wv h (no bias); q and k rotated by the position encoding; k and
v written to the token's row of the cache; query head h attends through KV head
h // (H/KVH) to the keys of its own sequence up to its own position (all of them, the last
`window`, or those of its own chunk of `chunk` positions); x += Wo o.  Reference: core/model.cpp:370-444 (decode) and :570-630
(prefill); here one code path serves both, reading keys and values from the cache.

The three projections are fused into one matrix product at load ([Wq; Wk; Wv]); an entry
that reads another entry's cache projects q only.  A position encoding that turns only part of
a head (parts/positions.py: `head_order`) has the rows of Wq and Wk reordered at load.
"""
from __future__ import annotations

import math

import torch

from ..csrc import ops
from .linear import chain_flags, matmul_nt
from .registry import MIXERS, Part
from .spec import TensorDecl, attention_cache_need, mask_span, visible_keys, visible_pairs

_NAMES = {"q": "self_attn.q_proj.weight", "k": "self_attn.k_proj.weight", "v": "self_attn.v_proj.weight",
          "o": "self_attn.o_proj.weight"}


@MIXERS.register("gqa_attention")
class GQAAttention(Part):
    graph_safe = True
    """params: hidden_size, num_heads, num_kv_heads, head_dim, position (a position
    encoding object or None), window (0 = all keys), chunk (0 = no chunks; not with a window),
    scale (default head_dim^-1/2), reads_cache (the layer has no key and value projections: it
    reads another entry's cache), tensor_names (optional overrides of q/k/v/o names under the prefix)."""

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.D = int(self._need("hidden_size"))
        self.H = int(self._need("num_heads"))
        self.KVH = int(self._need("num_kv_heads"))
        self.hd = int(self._need("head_dim"))
        if self.H % self.KVH:
            raise ValueError(f"gqa_attention: {self.H} heads are not a multiple of {self.KVH} KV heads")
        if self.hd % 2 or not 2 <= self.hd <= ops.MAX_HEAD_DIM:
            raise ValueError(f"gqa_attention: head_dim {self.hd} is outside what the attention kernels take "
                             f"(even, 2..{ops.MAX_HEAD_DIM})")
        self.span = mask_span(self.params.get("window"), self.params.get("chunk"))
        self.reads_cache = bool(self.params.get("reads_cache", False))
        self.scale = float(self.params.get("scale") or 1.0 / math.sqrt(self.hd))
        self.position = self.params.get("position")
        self.names = {k: prefix + v for k, v in {**_NAMES, **self.params.get("tensor_names", {})}.items()}
        self.w_qkv = self.w_o = None

    def tensors(self):
        q, kv = self.H * self.hd, self.KVH * self.hd
        own = [] if self.reads_cache else [TensorDecl(self.names["k"], (kv, self.D)),
                                           TensorDecl(self.names["v"], (kv, self.D))]
        return [TensorDecl(self.names["q"], (q, self.D))] + own + [TensorDecl(self.names["o"], (self.D, q))]

    def load(self, get):
        to = self.rt.to_compute
        order = getattr(self.position, "head_order", lambda: None)()
        if order is not None:
            order = torch.tensor(order, device=self.rt.device)

        def turned(name, heads):
            w = to(get(self.names[name]))
            return w if order is None else w.view(heads, self.hd, self.D)[:, order].reshape(heads * self.hd, self.D)
        parts = [turned("q", self.H)] + ([] if self.reads_cache else [turned("k", self.KVH), to(get(self.names["v"]))])
        self.w_qkv = torch.cat(parts, 0).contiguous()
        self.w_o = to(get(self.names["o"]))

    def cache_need(self):
        return attention_cache_need(self.KVH, self.hd, self.span)

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.w_qkv, self.w_o) if t is not None)

    def cache_bytes_per_query(self, context):
        return visible_keys(self.span, context) * 2 * self.KVH * self.hd * (2 if self.rt.dtype == torch.bfloat16 else 4)

    def flops(self, start, count):
        rows = 2 * self.H + (0 if self.reads_cache else 2 * self.KVH)            # q, k, v and o projections
        return count * 2.0 * self.D * rows * self.hd + \
            4.0 * self.H * self.hd * visible_pairs(self.span, start, count)      # q.k and p.v

    def first_weights(self):
        return self.w_qkv

    joint_weight = "w_qkv"         # parts/block.py: JoinedInput

    def forward(self, h, residual, ctx, cache, state, owns_cache=True, projected=None):
        """projected: Wqkv h (Wq h first), computed by the caller; the rotation works in it."""
        if self.reads_cache and owns_cache:
            raise ValueError("gqa_attention: a layer without key and value projections must read another entry's cache")
        T = h.shape[0]
        q_width = self.H * self.hd
        width = q_width + (2 * self.KVH * self.hd if owns_cache else 0)
        if projected is not None:
            qkv = projected[:, :width]
        else:
            qkv = self.rt.empty(T, width)
            # how the products are chained to their neighbours in the stream: parts/linear.py
            matmul_nt(self.rt, qkv, h, self.w_qkv[:width], early=chain_flags("mixer_in", T))
        cos, sin = self.position.tables() if self.position is not None else (None, None)
        from . import attention_dispatch as ad
        o = self.rt.empty(T, q_width)
        ad.mixer_core(self.rt, o, qkv, cos, sin, cache, ctx, self.H, self.KVH, self.hd, self.span, self.scale,
                      owns_cache)
        matmul_nt(self.rt, residual, o, self.w_o, accumulate=True, early=chain_flags("mixer_out", T),
                  then=self.rt.next_weights)
