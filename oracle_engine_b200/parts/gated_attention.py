"""Mixer `gated_attention`: grouped-query attention over the paged cache whose queries and keys are normed over the whole
projection, with a window and an output gate that reads the layer's input.

    q = Wq h [H dk], k = Wk h [G dk], v = Wv h [G dv]                                                     (no bias)
    q <- q / sqrt(mean(q^2) + eps) * wq over all H dk values at once, k likewise over its G dk, wk; then split into heads
    q, k: the first `dims` dimensions of each head turned by the token's position (the position encoding's cos/sin table),
          2i paired with 2i + 1 ("interleaved") or i with i + dims/2 ("halves"); the other dimensions pass
    s_j = scale * q . k_j for the keys pos - window < j <= pos (all j <= pos when window is 0);  softmax;  o = sum_j p_j v_j
    x += Wo (concat_heads(o) * sigmoid(Wg h))
Query head i reads key/value head i // (H / G).

One product makes [q | k | v | g] (csrc/attention_prep.cu: qkv_row_norm_rot_write norms and turns from it), the gate is
applied where the attention's result is stored.  The cache keeps per token "k" (G, dk), the normed and turned key, and
"v" (G, dv).
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .linear import chain_flags, matmul_nt
from .registry import MIXERS, Part
from .spec import TensorDecl, mask_span, span_need, visible_keys, visible_pairs

_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}


@MIXERS.register("gated_attention")
class GatedAttention(Part):
    graph_safe = True
    can_overwrite = True
    """params: hidden_size, num_heads, num_kv_heads, key_dim, value_dim, scale, eps, window (0 or None: all keys), chunk
    (chunks of positions instead of a window), position (a `rotary` encoding whose head_dim is the number of turned
    dimensions, or None), pairing ("interleaved", the default, or "halves"), tensor_names (optional overrides)."""

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.D = int(self._need("hidden_size"))
        self.H = int(self._need("num_heads"))
        self.G = int(self._need("num_kv_heads"))
        self.dk = int(self._need("key_dim"))
        self.dv = int(self._need("value_dim"))
        self.scale = float(self._need("scale"))
        self.eps = float(self._need("eps"))
        self.span = mask_span(self.params.get("window"), self.params.get("chunk"))
        self.position = self.params.get("position")
        self.pairing = self.params.get("pairing") or "interleaved"
        if self.H % self.G:
            raise ValueError(f"gated_attention: {self.H} heads are not a multiple of {self.G} key heads")
        if not (1 <= self.dk <= ops.MAX_HEAD_DIM and 1 <= self.dv <= ops.MAX_HEAD_DIM):
            raise ValueError(f"gated_attention: head sizes up to {ops.MAX_HEAD_DIM} are supported")
        if self.pairing not in ("interleaved", "halves"):
            raise ValueError("gated_attention: pairing is interleaved or halves")
        self.rot = 0 if self.position is None else int(self.position.head_dim)
        if self.rot % 2 or self.rot > self.dk:
            raise ValueError(f"gated_attention: {self.rot} turned dimensions must be even and at most key_dim {self.dk}")
        self.names = {k: prefix + v for k, v in {**_NAMES, **self.params.get("tensor_names", {})}.items()}
        self.w_in = self.w_o = self.norm_w = None

    def tensors(self):
        n, qw, kw, vw, ow = self.names, self.H * self.dk, self.G * self.dk, self.G * self.dv, self.H * self.dv
        return [TensorDecl(n["q"], (qw, self.D)), TensorDecl(n["k"], (kw, self.D)), TensorDecl(n["v"], (vw, self.D)),
                TensorDecl(n["q_norm"], (qw,), "ones_normal"), TensorDecl(n["k_norm"], (kw,), "ones_normal"),
                TensorDecl(n["g"], (ow, self.D)), TensorDecl(n["o"], (self.D, ow))]

    def load(self, get):
        to, f32, n = self.rt.to_compute, self.rt.to_f32, self.names
        self.w_in = torch.cat([to(get(n[k])) for k in ("q", "k", "v", "g")], 0).contiguous()
        self.w_o = to(get(n["o"]))
        self.norm_w = (f32(get(n["q_norm"])), f32(get(n["k_norm"])))

    def cache_need(self):
        return span_need((("k", (self.G, self.dk)), ("v", (self.G, self.dv))), self.span)

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_o) if t is not None)

    def cache_bytes_per_query(self, context):
        return visible_keys(self.span, context) * self.G * (self.dk + self.dv) * (2 if self.rt.dtype == torch.bfloat16 else 4)

    def flops(self, start, count):
        rows = (self.H + self.G) * (self.dk + self.dv) + self.H * self.dv
        return count * 2.0 * self.D * rows + 2.0 * self.H * (self.dk + self.dv) * visible_pairs(self.span, start, count)

    def first_weights(self):
        return self.w_in

    joint_weight = "w_in"          # parts/parallel.py: branches that read the same input

    def forward(self, h, residual, ctx, cache, state, owns_cache=True, overwrite: bool = False, projected=None):
        """overwrite: the output is written into `residual` (float32) instead of added.  projected: [q | k | v | g] h,
        computed by the caller; the queries are normed and turned in it."""
        if not owns_cache:
            raise ValueError("gated_attention: reading another entry's cache is not supported")
        T, H, G, dk, dv = h.shape[0], self.H, self.G, self.dk, self.dv
        proj = projected
        if proj is None:
            proj = self.rt.buffer("gatt.proj", T, self.w_in.shape[0])
            matmul_nt(self.rt, proj, h, self.w_in, early=chain_flags("mixer_in", T))
        kc, vc = cache.tensors["k"], cache.tensors["v"]
        ops.qkv_row_norm_rot_write(proj, kc, vc, self.norm_w, self.eps, self.position.tables() if self.rot else None,
                                   self.rot, self.pairing, cache.tables, ctx.tok_seq, ctx.tok_pos, H, G, dk, dv)
        o = self.rt.buffer("gatt.o", T, H * dv)
        off = H * dk + G * (dk + dv)
        from . import attention_dispatch as ad
        ad.split_attend(self.rt, o, proj, kc, vc, cache.tables, ctx, H, G, dk, dv, self.span, self.scale, 0.0,
                        gate=proj[:, off:off + H * dv])
        matmul_nt(self.rt, residual, o, self.w_o, accumulate=not overwrite, early=chain_flags("mixer_out", T))
