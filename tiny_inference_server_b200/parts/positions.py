"""Position encodings."""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from ..registry import register_part
from .base import BuildContext, PositionEncoding


class RotaryHalf(PositionEncoding):
    """Rotary encoding with the two halves of a head paired, (i, i + rot/2), as upstream
    (``precompute_rope_fast`` and ``rotate_half``, main_models_new.py:63-80):
    angle[pos, i] = pos * theta^(-2i/rot).  Tables of cos and sin, ``[positions, rot/2]``
    float32; the angles are formed in float64 on the host so that a table entry is the
    correctly rounded value.  ``factor`` divides every angle (positions interpolated linearly).  ``rotary_dim`` below the head size leaves the rest of each
    head unrotated; ``interleaved`` pairs (2i, 2i+1) instead."""

    def __init__(self, head_dim: int, theta: float, max_positions: int, rotary_dim: Optional[int] = None,
                 interleaved: bool = False, prefix: str = "", factor: float = 1.0):
        super().__init__(prefix)
        if not factor > 0:
            raise ValueError(f"a rotation's angles are divided by a positive number, not {factor}")
        self.factor = float(factor)
        self.head_dim = head_dim
        self.rotary_dim = head_dim if rotary_dim is None else rotary_dim
        if self.rotary_dim % 2 or not (0 < self.rotary_dim <= head_dim):
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {head_dim}")
        self.theta = float(theta)
        self.max_positions = max_positions
        self.interleaved = interleaved
        self.cos: Optional[torch.Tensor] = None
        self.sin: Optional[torch.Tensor] = None

    @classmethod
    def from_config(cls, cfg):
        return cls(cfg.head_dim, cfg.rope_theta, cfg.max_context)

    def tables(self):
        i = torch.arange(0, self.rotary_dim // 2, dtype=torch.float64)
        inv = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -2.0 * i / self.rotary_dim) / self.factor
        ang = torch.outer(torch.arange(self.max_positions, dtype=torch.float64), inv)
        return torch.cos(ang).to(torch.float32), torch.sin(ang).to(torch.float32)

    def load(self, tensors, ctx: BuildContext) -> None:
        cos, sin = self.tables()
        self.cos = cos.to(ctx.device).contiguous()
        self.sin = sin.to(ctx.device).contiguous()

    def encode_and_store(self, qkv, step, *, num_heads, kv_heads, head_dim, plane, block_table, page_size) -> None:
        """One kernel: rotate queries (in place) and keys in float32 and write keys and values of
        every row into its page (upstream does the three in turn: main_models_new.py:75-80,
        108-112)."""
        ops.rope_kv_write(qkv, step.positions, step.row_slot, self.cos, self.sin, plane, block_table, num_heads,
                          kv_heads, head_dim, page_size, step.fault, interleaved=self.interleaved,
                          write_kv=plane is not None)


    def fused_rotary(self):
        if self.interleaved or self.rotary_dim != self.head_dim:
            return None
        return self.cos, self.sin


class RotaryInterleaved(RotaryHalf):
    """Pairs (2i, 2i+1) instead of (i, i + rot/2); the same angles."""

    def __init__(self, head_dim: int, theta: float, max_positions: int, rotary_dim: Optional[int] = None,
                 prefix: str = "", factor: float = 1.0):
        super().__init__(head_dim, theta, max_positions, rotary_dim, interleaved=True, prefix=prefix, factor=factor)


class RotaryRescaled(RotaryHalf):
    """``RotaryHalf`` whose frequencies are rescaled for contexts longer than the ``original`` one a model was
    trained on.  With f_i = theta^(-2i/rot) and c(r) = rot * ln(original / (2 pi r)) / (2 ln theta) — the channel
    whose wave turns r times over the original context — channels up to lo = max(floor(c(fast)), 0) keep f_i,
    channels from hi = min(ceil(c(slow)), rot - 1) on use f_i / factor, and between them the two are blended with the
    weight clamp((i - lo) / max(hi - lo, 0.001), 0, 1); cosines and sines are multiplied by 0.1 ln(factor) + 1.
    ``scaling`` None: plain frequencies, magnitude 1.  The tables are formed in float64 on the host."""

    def __init__(self, head_dim: int, theta: float, max_positions: int, scaling: Optional[dict] = None,
                 rotary_dim: Optional[int] = None, prefix: str = ""):
        super().__init__(head_dim, theta, max_positions, rotary_dim, interleaved=False, prefix=prefix)
        self.scaling = dict(scaling) if scaling else None

    def frequencies(self):
        """(float64 frequencies (rot/2,), magnitude)."""
        import math
        rot = self.rotary_dim
        i = torch.arange(0, rot // 2, dtype=torch.float64)
        f = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -2.0 * i / rot)
        sc = self.scaling
        if not sc:
            return f, 1.0
        factor, original = float(sc["factor"]), float(sc["original"])

        def channel(turns: float) -> float:
            return rot * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.theta))

        lo = max(math.floor(channel(float(sc["fast"]))), 0)
        hi = min(math.ceil(channel(float(sc["slow"]))), rot - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0

    def tables(self):
        f, magnitude = self.frequencies()
        ang = torch.outer(torch.arange(self.max_positions, dtype=torch.float64), f)
        return (torch.cos(ang) * magnitude).to(torch.float32), (torch.sin(ang) * magnitude).to(torch.float32)

    def fused_rotary(self):
        return None


class RotaryBanded(RotaryInterleaved):
    """``RotaryInterleaved`` whose frequencies are slowed down by their wavelength, in three bands: with w = 2 pi / f, waves shorter
    than ``original / high`` keep f, those longer than ``original / low`` turn with f / factor, and between them the two are
    blended, ``(1 - s) f / factor + s f`` with ``s = (original / w - low) / (high - low)``.  ``scaling`` None: plain
    frequencies.  The tables are formed in float64 on the host."""

    def __init__(self, head_dim: int, theta: float, max_positions: int, scaling: Optional[dict] = None,
                 rotary_dim: Optional[int] = None, prefix: str = ""):
        super().__init__(head_dim, theta, max_positions, rotary_dim, prefix=prefix)
        self.scaling = dict(scaling) if scaling else None

    def frequencies(self) -> torch.Tensor:
        import math
        i = torch.arange(0, self.rotary_dim // 2, dtype=torch.float64)
        f = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -2.0 * i / self.rotary_dim)
        if not self.scaling:
            return f
        factor, low, high, original = (float(self.scaling[k]) for k in ("factor", "low", "high", "original"))
        turns = original * f / (2.0 * math.pi)              # of a wave over the original context
        s = (turns - low) / (high - low) if high != low else torch.zeros_like(f)
        blended = (1.0 - s) * f / factor + s * f
        return torch.where(turns > high, f, torch.where(turns < low, f / factor, blended))

    def tables(self):
        ang = torch.outer(torch.arange(self.max_positions, dtype=torch.float64), self.frequencies())
        return torch.cos(ang).to(torch.float32), torch.sin(ang).to(torch.float32)


register_part("position", "rope_banded", RotaryBanded)
register_part("position", "rope_half", RotaryHalf)
register_part("position", "rope_rescaled", RotaryRescaled)
register_part("position", "rope_interleaved", RotaryInterleaved)
