"""Position encodings.  `rotary`: rotate-half RoPE with optional llama3 or YaRN frequency scaling.

The reference computes theta_i = pos / base^(2i/hd) and its cosine and sine per token
(core/ops.cpp:461-466) and has no frequency scaling.  Here the inverse frequencies are
computed once on the host in double precision, scaled as config.json's `rope_scaling`
says, and turned into float32 cos/sin tables [max_positions, hd/2] that the kernels read.

llama3 scaling, with f_i = base^(-2i/hd) and wavelength l_i = 2 pi / f_i:
  l_i < orig/high_freq_factor          keep f_i
  l_i > orig/low_freq_factor           f_i / factor
  otherwise  s = (orig/l_i - low)/(high - low);  f_i' = (1-s) f_i/factor + s f_i

YaRN scaling (`kind` "yarn"), with c(t) = dims ln(orig / (2 pi t)) / (2 ln base), the pair that makes t turns over orig
positions:  lo = max(floor c(fast), 0), hi = min(ceil c(slow), dims - 1), r_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1),
f_i' = r_i f_i / factor + (1 - r_i) f_i, and cosine and sine are multiplied by 0.1 ln(factor) + 1.
"""
from __future__ import annotations

import math

import torch

from .registry import POSITIONS, Part


def rotary_inv_freq(head_dim: int, theta: float, scaling: dict | None) -> torch.Tensor:
    half = head_dim // 2
    f = torch.tensor([theta ** (-(2.0 * i) / head_dim) for i in range(half)], dtype=torch.float64)
    if not scaling:
        return f
    factor = float(scaling["factor"])
    if scaling.get("kind") == "yarn":
        r = _yarn_ramp(head_dim, theta, scaling)
        return f / factor * r + f * (1.0 - r)
    low = float(scaling["low_freq_factor"])
    high = float(scaling["high_freq_factor"])
    orig = float(scaling["original_max_position_embeddings"])
    out = f.clone()
    for i in range(half):
        fi = f[i].item()
        wavelen = 2.0 * math.pi / fi
        if wavelen < orig / high:
            continue
        if wavelen > orig / low:
            out[i] = fi / factor
        else:
            s = (orig / wavelen - low) / (high - low)
            out[i] = (1.0 - s) * fi / factor + s * fi
    return out


def _yarn_ramp(dims: int, theta: float, scaling: dict) -> torch.Tensor:
    orig = float(scaling["original"])

    def pair(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
    lo = max(math.floor(pair(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair(float(scaling["slow"]))), dims - 1)
    i = torch.arange(dims // 2, dtype=torch.float64)
    return ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)


def rotary_magnitude(scaling: dict | None) -> float:
    """What cosine and sine are multiplied by."""
    return 0.1 * math.log(float(scaling["factor"])) + 1.0 if scaling and scaling.get("kind") == "yarn" else 1.0


@POSITIONS.register("rotary")
class Rotary(Part):
    """params: head_dim, theta, scaling (None, the llama3 dict or the YaRN one: "kind" "yarn", factor, original, fast,
    slow), max_positions, dims (how many dimensions of a head are
    turned, at frequencies theta^(-2i/dims); default head_dim).  With dims < head_dim the tables still have head_dim / 2
    columns, the ones behind dims / 2 at angle zero (`head_order` says which dimensions a mixer puts there)."""

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.head_dim = int(self._need("head_dim"))
        if self.head_dim % 2:
            raise ValueError(f"rotary: head_dim {self.head_dim} must be even")
        self.dims = int(self.params.get("dims", self.head_dim))
        if self.dims % 2 or not 0 <= self.dims <= self.head_dim:
            raise ValueError(f"rotary: {self.dims} turned dimensions must be even and at most head_dim {self.head_dim}")
        self.max_positions = int(self._need("max_positions"))
        self.inv_freq = rotary_inv_freq(self.dims, float(self._need("theta")), self.params.get("scaling"))
        self.magnitude = rotary_magnitude(self.params.get("scaling"))
        self.cos = self.sin = None

    def tables(self):
        """(cos, sin), float32 [max_positions, head_dim/2] on the device."""
        if self.cos is None:
            pos = torch.arange(self.max_positions, dtype=torch.float64)
            freq = torch.cat([self.inv_freq, torch.zeros((self.head_dim - self.dims) // 2, dtype=torch.float64)])
            ang = pos[:, None] * freq[None, :]
            self.cos = (torch.cos(ang) * self.magnitude).to(torch.float32).to(self.rt.device).contiguous()
            self.sin = (torch.sin(ang) * self.magnitude).to(torch.float32).to(self.rt.device).contiguous()
        return self.cos, self.sin

    def head_order(self) -> list | None:
        """None, or, when only the first `dims` dimensions of a head are turned (i paired with i + dims/2), the order
        that puts every turned pair at (j, j + head_dim/2) and the untouched dimensions, in pairs of angle zero, behind
        them: kernels that rotate whole heads by halves then rotate exactly the first `dims`.  A score is a sum over
        the dimensions, so a query and a key that are both kept in this order score as before."""
        if self.dims == self.head_dim:
            return None
        if self.magnitude != 1.0:
            raise ValueError("rotary: dimensions at angle zero would take the scaling's magnitude")
        r, half = self.dims // 2, self.head_dim // 2
        rest = list(range(self.dims, self.head_dim))
        return list(range(r)) + rest[:half - r] + list(range(r, self.dims)) + rest[half - r:]


@POSITIONS.register("rotary_pairs")
class RotaryPairs(Part):
    """Rotation of the pairs (2i, 2i+1), i < dims/2, of a head by position * base^(-2i/dims); dimensions
    from `dims` on pass unchanged.  No table and no largest position: the kernel forms the angle as
    float32(position) * float32(frequency) and takes its sine and cosine in float32.
    params: dims, base."""

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.dims = int(self._need("dims"))
        self.base = float(self._need("base"))
        if self.dims % 2 or self.dims < 0:
            raise ValueError(f"rotary_pairs: dims {self.dims} must be even")
        self.inv_freq = None

    def tables(self):
        """(frequencies float32 [dims/2] on the device, dims)."""
        if self.inv_freq is None:
            f = [self.base ** (-(2.0 * i) / self.dims) for i in range(self.dims // 2)]
            self.inv_freq = torch.tensor(f or [0.0], dtype=torch.float64).to(torch.float32).to(self.rt.device)
        return self.inv_freq, self.dims


@POSITIONS.register("none")
class NoPosition(Part):
    """No position encoding: queries and keys are used as projected."""

    def tables(self):
        return None, None
