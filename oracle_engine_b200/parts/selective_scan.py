"""Mixer `selective_scan`: a recurrent layer with a state of N values per channel whose decay, input and read-out depend on
the token.

    [x | z] = Win h  (C channels each);   u = silu(conv(x) + cb): causal convolution over time, per channel
    [r | b | c] = Wx u  (rank, N, N values);   dt = softplus(Wdt r + db)  (C values);   A = -exp(A_log)  [C, N]
    S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c b_n;   y_c = sum_n S[c, n] c_n + D_c u_c;     S starts at zero
    out += Wo (y * silu(z))
b, c, dt, the decays and S are float32 on both paths; u, like every projection, is of the compute type.  S and the
convolution's last taps - 1 inputs are per-sequence state (float32).

A step of one token per sequence takes three kernels between the input and the output product: the convolution (which moves
its state on), the thin product Wx u and the scan with the step sizes' product inside.  Other steps make the step sizes by
a product of their own; the bfloat16 path runs long prompts as segments side by side (csrc/selective_scan.cu).
"""
from __future__ import annotations

import math

import torch

from ..csrc import ops
from .linear import chain_flags, matmul_nt
from .registry import MIXERS, Part
from .spec import StateNeed, TensorDecl

_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "x": "x", "dt": "dt", "dt_bias": "dt.b", "A_log": "A_log",
          "D": "D", "o": "o"}

SEGMENTS_FROM = 128         # a step whose longest sequence brings this many tokens runs them as segments side by side
SEGMENT_MIN = 32            # tokens of the shortest segment
SEGMENT_THREADS = 148 * 1024     # threads of the scan that keep the GPU busy


def segment_plan(C: int, N: int, n_seqs: int, longest: int) -> tuple | None:
    """(tokens of a segment, segments a sequence) for a step whose longest sequence brings `longest` tokens, or None."""
    lanes = -(-N // 16)
    n_seg = max(1, min(-(-SEGMENT_THREADS // (C * lanes * max(1, n_seqs))), longest // SEGMENT_MIN))
    seg_len = -(-(-(-longest // n_seg)) // 8) * 8
    n_seg = -(-longest // seg_len)
    return None if n_seg < 2 else (seg_len, n_seg)


@MIXERS.register("selective_scan")
class SelectiveScan(Part):
    graph_safe = True
    can_overwrite = True
    """params: hidden_size, inner (C), state (N), dt_rank, conv_taps, tensor_names (optional overrides)."""

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.D = int(self._need("hidden_size"))
        self.C = int(self._need("inner"))
        self.N = int(self._need("state"))
        self.rank = int(self._need("dt_rank"))
        self.taps = int(self._need("conv_taps"))
        if not (1 <= self.N <= 256 and 1 <= self.taps <= 32):
            raise ValueError("selective_scan: up to 256 states per channel and 1..32 taps are supported")
        self.ldw = -(-self.rank // 8) * 8          # columns of Wdt as kept, zeros behind the rank: 16-byte rows
        self.names = {k: prefix + v for k, v in {**_NAMES, **self.params.get("tensor_names", {})}.items()}
        self.w_in = self.w_x = self.w_dt = self.w_o = None

    def tensors(self):
        n, C, N = self.names, self.C, self.N
        return [TensorDecl(n["in"], (2 * C, self.D)), TensorDecl(n["conv"], (C, self.taps)), TensorDecl(n["conv_bias"], (C,)),
                TensorDecl(n["x"], (self.rank + 2 * N, C)), TensorDecl(n["dt"], (C, self.rank)),
                TensorDecl(n["dt_bias"], (C,)), TensorDecl(n["A_log"], (C, N)), TensorDecl(n["D"], (C,), "ones_normal"),
                TensorDecl(n["o"], (self.D, C))]

    def load(self, get):
        to, f32, n = self.rt.to_compute, self.rt.to_f32, self.names
        pad = self.ldw - self.rank
        self.w_in, self.w_o = to(get(n["in"])), to(get(n["o"]))
        # rows of zeros behind the rank: the thin product leaves zeros there, and b and c start on 16-byte boundaries
        wx = to(get(n["x"]))
        self.w_x = torch.cat([wx[:self.rank], wx.new_zeros(pad, self.C), wx[self.rank:]], 0).contiguous()
        self.w_dt = torch.nn.functional.pad(to(get(n["dt"])), (0, pad)).contiguous()
        self.conv_w, self.conv_b = f32(get(n["conv"])).T.contiguous(), f32(get(n["conv_bias"]))
        self.dt_bias, self.skip = f32(get(n["dt_bias"])), f32(get(n["D"]))
        self.A2 = (-torch.exp(f32(get(n["A_log"])).double()) * math.log2(math.e)).float().contiguous()

    def state_need(self):
        return {"S": StateNeed((self.C, self.N), torch.float32),
                "conv": StateNeed((max(self.taps - 1, 1), self.C), torch.float32)}

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_x, self.w_dt, self.w_o) if t is not None) + \
            (0 if self.w_in is None else 4 * self.C * (self.N + self.taps + 3))

    def cache_bytes_per_query(self, context):
        return 2 * 4 * self.C * (self.N + max(self.taps - 1, 1))          # the state, read and written

    def flops(self, start, count):
        return count * 2.0 * (3 * self.D * self.C + self.C * (2 * self.rank + 2 * self.N) + 3 * self.C * self.N)

    def first_weights(self):
        return self.w_in

    joint_weight = "w_in"          # parts/parallel.py: branches that read the same input

    def _segments(self, ctx):
        """How a step with long prompts cuts its sequences into segments that run side by side, or None for the one walk.
        float32 serving keeps the one walk: there a position's logits are the same bits under every cut of the prompt."""
        longest = int(ctx.max_qlen)
        if self.rt.dtype != torch.bfloat16 or longest < SEGMENTS_FROM or torch.cuda.is_current_stream_capturing():
            return None             # (a captured step's longest sequence is a bound, not a length)
        plan = segment_plan(self.C, self.N, ctx.n_seqs, longest)
        if plan is None:
            return None
        seg_len, n_seg = plan
        seg_state = self.rt.buffer("ssm.seg_state", ctx.n_seqs * n_seg, self.C * self.N, dtype=torch.float32)
        seg_dt = self.rt.buffer("ssm.seg_dt", ctx.n_seqs * n_seg, self.C, dtype=torch.float32)
        return seg_len, n_seg, seg_state, seg_dt

    def forward(self, h, residual, ctx, cache, state, owns_cache=True, overwrite: bool = False, projected=None):
        """overwrite: the output is written into `residual` (float32) instead of added.  projected: [x | z] = Win h, computed
        by the caller."""
        T, f32, buf, C = h.shape[0], torch.float32, self.rt.buffer, self.C
        xz = projected
        if xz is None:
            xz = buf("ssm.in", T, 2 * C)
            matmul_nt(self.rt, xz, h, self.w_in, early=chain_flags("mixer_in", T))
        u = buf("ssm.u", T, C)
        ops.causal_conv(u, xz[:, :C], self.conv_w, self.conv_b, state["conv"], ctx)
        thin = buf("ssm.thin", T, self.ldw + 2 * self.N, dtype=f32)
        matmul_nt(self.rt, thin, u, self.w_x)
        y = buf("ssm.y", T, C)
        z, off_b, off_c = xz[:, C:2 * C], self.ldw, self.ldw + self.N
        # float32 serving makes the step sizes the one way, so that a position's logits are the same bits under every cut
        if self.rt.dtype != f32 and ctx.all_decode and ctx.n_tokens == ctx.n_seqs:
            ops.selective_step(y, state["S"], u, self.w_dt, 0, self.rank, self.dt_bias, thin, off_b, off_c, self.A2, self.skip,
                               z, ctx)
        else:
            low = thin[:, :self.ldw]
            if self.rt.dtype != f32:
                low = buf("ssm.low", T, self.ldw)           # the second thin product's operand, in the compute dtype
                ops.thin_cast(low, thin)
            zdt = buf("ssm.zdt", T, C, dtype=f32)
            matmul_nt(self.rt, zdt, low, self.w_dt)
            ops.selective_scan(y, state["S"], u, zdt, self.dt_bias, thin, off_b, off_c, self.A2, self.skip, z, ctx,
                               segments=self._segments(ctx))
        matmul_nt(self.rt, residual, y, self.w_o, accumulate=not overwrite, early=chain_flags("mixer_out", T))
