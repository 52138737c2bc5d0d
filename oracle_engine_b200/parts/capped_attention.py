"""Mixer `capped_attention`: grouped-query attention over the paged cache whose keys and values have head sizes of
their own, with a partial rotation, a cap on the scores and an optional window or chunks.

    q = Wq h [H, dk], k = Wk h [G, dk], v = Wv h [G, dv]                    (no bias)
    q, k: the first `rot` dimensions of each head turned by the token's position, dimension i < rot/2 paired with
          i + rot/2 (the position encoding's cos/sin table [positions, rot/2]); the other dimensions pass
    s_j = scale * q . k_j;  s_j <- cap * tanh(s_j / cap) if cap > 0;  keys pos - window < j <= pos (with chunks
          those of pos's own chunk, with neither all j <= pos);  softmax over those keys;  x += Wo concat_heads(sum_j p_j v_j)
Query head i reads key/value head i // (H / G).

The cache keeps per token two tensors: "k" (G, dk), the turned key, and "v" (G, dv).  A layer with
`reads_cache` has no Wk and Wv: it reads the rows that another entry wrote for the same tokens.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .linear import matmul_nt
from .registry import MIXERS, Part
from .spec import TensorDecl, mask_span, span_need, visible_keys, visible_pairs

_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o"}


@MIXERS.register("capped_attention")
class CappedAttention(Part):
    graph_safe = True
    can_overwrite = True
    """params: hidden_size, num_heads, num_kv_heads, key_dim, value_dim, scale, softcap (0 or None: no cap),
    window (0 or None: all keys), chunk (0 or None: no chunks; not with a window), reads_cache (no Wk and Wv), position
    (a `rotary` encoding whose head_dim is the number of turned dimensions, or None), tensor_names (optional overrides)."""

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.D = int(self._need("hidden_size"))
        self.H = int(self._need("num_heads"))
        self.G = int(self._need("num_kv_heads"))
        self.dk = int(self._need("key_dim"))
        self.dv = int(self._need("value_dim"))
        self.scale = float(self._need("scale"))
        self.cap = float(self.params.get("softcap") or 0.0)
        self.span = mask_span(self.params.get("window"), self.params.get("chunk"))
        self.reads_cache = bool(self.params.get("reads_cache", False))
        self.position = self.params.get("position")
        if self.H % self.G:
            raise ValueError(f"capped_attention: {self.H} heads are not a multiple of {self.G} key heads")
        if not (1 <= self.dk <= ops.MAX_HEAD_DIM and 1 <= self.dv <= ops.MAX_HEAD_DIM):
            raise ValueError(f"capped_attention: head sizes up to {ops.MAX_HEAD_DIM} are supported")
        self.rot = 0 if self.position is None else int(self.position.head_dim)
        if self.rot % 2 or self.rot > self.dk:
            raise ValueError(f"capped_attention: {self.rot} turned dimensions must be even and at most key_dim {self.dk}")
        self.names = {k: prefix + v for k, v in {**_NAMES, **self.params.get("tensor_names", {})}.items()}
        self.w_qkv = self.w_o = None

    def tensors(self):
        n = self.names
        own = [] if self.reads_cache else [TensorDecl(n["k"], (self.G * self.dk, self.D)),
                                           TensorDecl(n["v"], (self.G * self.dv, self.D))]
        return [TensorDecl(n["q"], (self.H * self.dk, self.D))] + own + [TensorDecl(n["o"], (self.D, self.H * self.dv))]

    def load(self, get):
        to, n = self.rt.to_compute, self.names
        self.w_qkv = torch.cat([to(get(n[k])) for k in (("q",) if self.reads_cache else ("q", "k", "v"))], 0).contiguous()
        self.w_o = to(get(n["o"]))

    def cache_need(self):
        return span_need((("k", (self.G, self.dk)), ("v", (self.G, self.dv))), self.span)

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.w_qkv, self.w_o) if t is not None)

    def cache_bytes_per_query(self, context):
        return visible_keys(self.span, context) * self.G * (self.dk + self.dv) * (2 if self.rt.dtype == torch.bfloat16 else 4)

    def flops(self, start, count):
        rows = (self.H + (0 if self.reads_cache else self.G)) * (self.dk + self.dv)
        return count * 2.0 * self.D * rows + 2.0 * self.H * (self.dk + self.dv) * visible_pairs(self.span, start, count)

    def first_weights(self):
        return self.w_qkv

    joint_weight = "w_qkv"         # parts/block.py: JoinedInput

    def forward(self, h, residual, ctx, cache, state, owns_cache=True, overwrite: bool = False, projected=None):
        """overwrite: the output is written into `residual` (float32) instead of added.  projected: Wqkv h (Wq h first),
        computed by the caller; the rotation works in it."""
        if owns_cache == self.reads_cache:
            raise ValueError("capped_attention: a layer without key and value projections must read another entry's "
                             "cache (and one with them must own its cache)")
        T = h.shape[0]
        qw = self.H * self.dk
        qkv = projected
        if qkv is None:
            qkv = self.rt.buffer("capped.qkv", T, self.w_qkv.shape[0])
            matmul_nt(self.rt, qkv, h, self.w_qkv)
        cos, sin = self.position.tables() if self.rot else (None, None)
        kc, vc = cache.tensors["k"], cache.tensors["v"]
        o = self.rt.buffer("capped.o", T, self.H * self.dv)
        from . import attention_dispatch as ad
        ad.split_mixer_core(self.rt, o, qkv, cos, sin, self.rot, kc, vc, cache.tables, ctx, self.H, self.G, self.dk,
                            self.dv, self.span, self.scale, self.cap, owns_cache)
        matmul_nt(self.rt, residual, o, self.w_o, accumulate=not overwrite)
