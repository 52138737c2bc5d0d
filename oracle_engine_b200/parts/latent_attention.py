"""Mixer `latent_attention`: attention whose keys and values are projections of one small latent per token, so
that the latent (and one shared, turned key part) is all the cache keeps.

    q_h = (Wq h)_h                                      or, with a query latent (q_rank),  (Wuq (R(Wdq h) * wq))_h
          laid out per head as [dk dimensions without position | rd turned dimensions]
    d = Wdkv h:  c = R(d[:r]) * wc  (the latent),  kr = turn(d[r:], position)  (rd values shared by all heads)
    k_h,j = [Wuk_h c_j | kr_j],  v_h,j = Wuv_h c_j,  s_j = scale * q_h . k_h,j for j <= t,  softmax,  o_h = sum_j p_j v_h,j
    x += Wo (concat_h o_h [* sigmoid(Wg h)])                 the gate has one value per output or one per head
R(u) = u / sqrt(mean(u^2) + eps); turn: pairs (2i, 2i + 1), i < dims/2, by the angle position * base^(-2i/dims), or, with
a `rotary` encoding, by its cos/sin table (whose frequencies and magnitude may be rescaled), interleaved or halves paired.
Optional: a window (keys t - window < j <= t) or chunks; a sink, exp(sink_h) in the softmax's denominator without a key.

How it is computed: keys and values are never expanded.  The query goes through the key projection first,
qa_h = Wuk_h^T q_h[:dk] (r values), so that s_j = scale * (qa_h . c_j + turn(q_h[dk:]) . kr_j) reads the cache rows
[c_j | kr_j] directly, the same rows for every head; the heads' sums u_h = sum_j p_j c_j (r values) go through the
value projection afterwards, o_h = Wuv_h u_h (a gate per head multiplies u_h, which comes to the same).  A prompt, a piece of one and a decoded token take the same path.
A layer with `cache_from` in its schedule entry has no Wdkv: it reads the rows another layer wrote for the same
tokens, with projections of its own.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .linear import chain_flags, matmul_nt
from .registry import MIXERS, Part
from .spec import TensorDecl, mask_span, span_need, visible_keys, visible_pairs

_NAMES = {"q": "q", "dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk",
          "uv": "uv", "g": "g", "o": "o", "sink": "sink"}
HEAD_MATMUL_MAX_TOKENS = 16       # up to here the per-head products run as one launch that streams the weights once


@MIXERS.register("latent_attention")
class LatentAttention(Part):
    graph_safe = True
    can_overwrite = True
    """params: hidden_size, num_heads, key_dim (per head, without position), value_dim, kv_rank, scale, eps,
    rot_dim (0 or None: no turned part), position (a `rotary_pairs` encoding, or a `rotary` one whose head_dim is the number
    of turned dimensions; up to rot_dim), pairing (of a `rotary` encoding: "halves", the default, or "interleaved"), q_rank
    (0 or None: queries straight from the input), gate (True: a sigmoid output gate; "head": one value per head),
    window (0 or None: every key), chunk (chunks of positions instead), sink (True: a learned score per head joins the
    denominator), reads_cache (the layer owns no down projection: it reads another entry's cache), joined (True: one
    product of the compute type makes [queries | latent and turned part | gate per head]; not with q_rank or a gate per
    output, default False: what is normed or gated leaves its product in float32), tensor_names (optional overrides)."""

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.D = int(self._need("hidden_size"))
        self.H = int(self._need("num_heads"))
        self.dk = int(self._need("key_dim"))
        self.dv = int(self._need("value_dim"))
        self.r = int(self._need("kv_rank"))
        self.scale = float(self._need("scale"))
        self.eps = float(self._need("eps"))
        self.rd = int(self.params.get("rot_dim") or 0)
        self.q_rank = int(self.params.get("q_rank") or 0)
        self.gate = bool(self.params.get("gate", False))
        self.head_gate = self.params.get("gate") == "head"
        self.span = mask_span(self.params.get("window"), self.params.get("chunk"))
        self.sink = bool(self.params.get("sink", False))
        self.joined = bool(self.params.get("joined", False))
        self.pairing = self.params.get("pairing") or "halves"
        self.reads_cache = bool(self.params.get("reads_cache", False))
        self.position = self.params.get("position") if self.rd else None
        self.dims = 0 if self.position is None else int(self.position.dims)
        self.rotates_by_table = self.position is not None and self.position.kind == "rotary"
        if self.joined and (self.q_rank or (self.gate and not self.head_gate)):
            raise ValueError("latent_attention: one product for all takes no query latent and no gate per output")
        if self.dims > self.rd:
            raise ValueError(f"latent_attention: {self.dims} turned dimensions exceed rot_dim {self.rd}")
        if not 1 <= self.r <= 512:
            raise ValueError("latent_attention: kv_rank up to 512 is supported")
        self.names = {k: prefix + v for k, v in {**_NAMES, **self.params.get("tensor_names", {})}.items()}
        self.w = {}
        self.sinks = None

    @property
    def R(self):
        return self.r + self.rd

    @property
    def gate_rows(self):
        return 0 if not self.gate else self.H if self.head_gate else self.H * self.dv

    def tensors(self):
        n, qd = self.names, self.H * (self.dk + self.rd)
        out = []
        if self.q_rank:
            out += [TensorDecl(n["dq"], (self.q_rank, self.D)), TensorDecl(n["dq_norm"], (self.q_rank,), "ones_normal"),
                    TensorDecl(n["uq"], (qd, self.q_rank))]
        else:
            out.append(TensorDecl(n["q"], (qd, self.D)))
        if not self.reads_cache:
            out += [TensorDecl(n["dkv"], (self.R, self.D)), TensorDecl(n["dkv_norm"], (self.r,), "ones_normal")]
        out += [TensorDecl(n["uk"], (self.H * self.dk, self.r)), TensorDecl(n["uv"], (self.H * self.dv, self.r))]
        if self.gate:
            out.append(TensorDecl(n["g"], (self.gate_rows, self.D)))
        if self.sink:
            out.append(TensorDecl(n["sink"], (self.H,)))
        out.append(TensorDecl(n["o"], (self.D, self.H * self.dv)))
        return out

    def load(self, get):
        to, f32, n = self.rt.to_compute, self.rt.to_f32, self.names
        w = {}
        # one product with float32 output for everything that is normed, turned or gated in float32: [dq | dkv | g]; or,
        # `joined`, one of the compute type for [q | dkv | g]
        first = []
        if self.q_rank:
            first.append(to(get(n["dq"])))
            w["uq"] = to(get(n["uq"]))
            self.dq_norm = f32(get(n["dq_norm"]))
        elif self.joined:
            first.append(to(get(n["q"])))
        else:
            w["q"] = to(get(n["q"]))
        if self.sink:
            self.sinks = f32(get(n["sink"]))
        self.off_dkv = sum(t.shape[0] for t in first)
        if not self.reads_cache:
            first.append(to(get(n["dkv"])))
            self.dkv_norm = f32(get(n["dkv_norm"]))
        self.off_g = sum(t.shape[0] for t in first)
        if self.gate:
            first.append(to(get(n["g"])))
        if first:
            if self.joined and (rest := -sum(t.shape[0] for t in first) % 8):      # rows of 16-byte pieces: the products
                first.append(torch.zeros_like(first[0][:1]).expand(rest, -1))      # that read the queries take no others
            w["in"] = torch.cat(first, 0).contiguous()
        uk = to(get(n["uk"])).reshape(self.H, self.dk, self.r)
        w["uk_t"] = uk.transpose(1, 2).contiguous()                       # [H, r, dk]: qa_h = uk_t[h] @ q_h
        w["uv"] = to(get(n["uv"])).reshape(self.H, self.dv, self.r).contiguous()      # [H, dv, r]: o_h = uv[h] @ u_h
        w["o"] = to(get(n["o"]))
        self.w = w

    def cache_need(self):
        return span_need((("latent", (self.R,)),), self.span)

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in self.w.values())

    def cache_bytes_per_query(self, context):
        return visible_keys(self.span, context) * self.R * (2 if self.rt.dtype == torch.bfloat16 else 4)

    def flops(self, start, count):
        qd = self.H * (self.dk + self.rd)
        products = 2.0 * self.D * ((self.q_rank or qd) + (0 if self.reads_cache else self.R) +
                                   self.gate_rows + self.H * self.dv)
        products += 2.0 * self.q_rank * qd + 2.0 * self.H * self.r * (self.dk + self.dv)
        return count * products + 2.0 * self.H * (self.R + self.r) * visible_pairs(self.span, start, count)

    def first_weights(self):
        return self.w.get("in") if self.w.get("in") is not None else self.w.get("q")

    def _per_head(self, out, a, w):
        """out[:, h, :] = w[h] @ a[:, h, :].  bfloat16: one launch for all heads, a kernel that streams the weights once
        for a handful of tokens, the tensor cores for more; else a product per head (float32: the CUDA-core product
        whose sums do not depend on the batch)."""
        T = a.shape[0]
        if self.rt.dtype == torch.bfloat16 and T <= HEAD_MATMUL_MAX_TOKENS:
            ops.head_matmul(out, a, w)
            return
        if self.rt.dtype == torch.bfloat16 and self.rt.tensor_cores:
            from ..csrc import ops_tc
            if ops_tc.head_matmul_supported(a, w, out):
                ops_tc.head_matmul(out, a, w)
                return
        for h in range(self.H):
            matmul_nt(self.rt, out[:, h, :], a[:, h, :], w[h])

    def forward(self, h, residual, ctx, cache, state, owns_cache=True, overwrite: bool = False):
        """overwrite: the output is written into `residual` (float32) instead of added."""
        if owns_cache == self.reads_cache:
            raise ValueError("latent_attention: a layer without a down projection must read another entry's cache "
                             "(and one with it must own its cache)")
        T, f32, buf = h.shape[0], torch.float32, self.rt.buffer
        H, dk, dv, r, rd, R = self.H, self.dk, self.dv, self.r, self.rd, self.R
        qd = H * (dk + rd)
        proj = None
        if "in" in self.w:
            proj = buf("latent.in", T, self.w["in"].shape[0], dtype=None if self.joined else f32)
            matmul_nt(self.rt, proj, h, self.w["in"], early=chain_flags("mixer_in", T) if self.joined else 0)
        q = proj[:, :qd] if self.joined else buf("latent.q", T, qd)
        if self.joined:
            pass
        elif self.q_rank:
            cq = buf("latent.cq", T, self.q_rank)
            ops.group_rmsnorm(cq, proj[:, :self.q_rank], self.dq_norm, self.eps, 1)
            matmul_nt(self.rt, q, cq, self.w["uq"])
        else:
            matmul_nt(self.rt, q, h, self.w["q"])
        qfull = buf("latent.qfull", T, H * R)
        angles = {"freq": None}
        if self.rotates_by_table:
            angles.update(tables_cs=self.position.tables(), halves=self.pairing == "halves")
        elif self.dims:
            angles["freq"] = self.position.tables()[0]
        rows = cache.tensors["latent"]
        ops.latent_write(None if self.reads_cache else proj[:, self.off_dkv:self.off_dkv + R],
                         None if self.reads_cache else self.dkv_norm, self.eps, q, qfull, dims=self.dims,
                         cache=rows, tables=cache.tables, ctx=ctx, heads=H, dk=dk, r=r, rd=rd, write_cache=owns_cache,
                         **angles)
        self._per_head(qfull.view(T, H, R)[:, :, :r], q.unflatten(1, (H, dk + rd))[:, :, :dk], self.w["uk_t"])
        u = buf("latent.u", T, H * r)
        from . import attention_dispatch as ad
        gate = None
        if self.head_gate:
            gate = proj[:, self.off_g:self.off_g + H]
            if gate.dtype != u.dtype:
                raise ValueError("latent_attention: a gate per head goes with `joined` projections")
        ad.latent_core(self.rt, u, qfull, rows, cache.tables, ctx, H, r, rd, self.scale, self.span, self.sinks, gate)
        # with a gate the heads' outputs stay float32 until the gate has been applied
        late_gate = self.gate and not self.head_gate
        o = buf("latent.o", T, H * dv, dtype=f32 if late_gate else None)
        self._per_head(o.view(T, H, dv), u.view(T, H, r), self.w["uv"])
        if late_gate:
            y = buf("latent.y", T, H * dv)
            ops.head_gate(y, o, proj[:, self.off_g:self.off_g + H * dv], None, H, dv, False, "sigmoid")
            o = y
        matmul_nt(self.rt, residual, o, self.w["o"], accumulate=not overwrite)
