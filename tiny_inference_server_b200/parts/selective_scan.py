"""A selective scan (Mamba's first form): a recurrent mixer with a decay per channel and state."""
from __future__ import annotations

from typing import Dict

import torch

from ..kernels import ops, segment_plan
from ..registry import register_part
from .base import BuildContext, LayerBinding, Mixer, StateSpec, WeightSpec
from .short_conv import CausalConv
from .window_attention import pad8


class SelectiveScan(Mixer):
    """``inner`` channels with a state of ``state_dim`` numbers each (float32, zero at the start of a sequence):

    * ``W_in h`` is ``[x: inner | z: inner]``; x passes a short causal convolution per channel (``conv``, with bias ``conv.b``)
      and silu;
    * ``W_x x`` is ``[low: dt_rank | B: state_dim | C: state_dim]``; ``dt = softplus(W_dt low + dt.b)``, one per channel;
    * per channel c and state n, with ``A = -exp(A_log)``: ``S <- exp(dt A) S + dt x B_n``, ``y = sum_n S C_n + D x``;
    * ``y * silu(z)``, then ``W_o``.

    Tensor names below the prefix: ``in, x, dt, o`` (stored (out, in)), ``conv, conv.b``, ``dt.b``, ``A_log`` (inner, state_dim),
    ``D``.  The step sizes (their projection leaves its product in 32-bit), the decays, the state, the recurrence and the
    gate are 32-bit.  The state of a request is S of every channel followed by the convolution's last inputs."""

    graph_safe = True
    fuses_residual = True

    def __init__(self, width: int, inner: int, state_dim: int, dt_rank: int, conv_taps: int, prefix: str = ""):
        super().__init__(prefix)
        self.width, self.inner, self.state_dim, self.dt_rank = width, inner, state_dim, dt_rank
        self.conv = CausalConv([inner], conv_taps, ["conv"], prefix=prefix, silu=True, bias_name="conv.b")
        self.z_at = pad8(inner)
        self.b_at = pad8(dt_rank)
        self.c_at = self.b_at + pad8(state_dim)
        self.state_floats = inner * state_dim
        self.w_in = self.w_x = self.w_dt = self.w_o = self.dt_bias = self.a_log = self.skip = None

    @classmethod
    def from_config(cls, cfg, prefix: str, layer_index: int, lag: int = 0, position=None):
        m = cfg.layers[layer_index]["mixer"]
        return cls(cfg.hidden_size, m["inner"], m["state"], m["dt_rank"], m["conv"], prefix=prefix)

    def children(self):
        return (self.conv,)

    def step_planners(self):
        return (segment_plan.planner(),)

    def state_spec(self) -> StateSpec:
        return StateSpec((self.state_floats + self.conv.state_floats,), torch.float32)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        i, n = self.inner, self.state_dim
        return {"in": WeightSpec((2 * i, self.width)), "x": WeightSpec((self.dt_rank + 2 * n, i)),
                "dt": WeightSpec((i, self.dt_rank)), "dt.b": WeightSpec((i,), init="uniform", lo=-4.0, hi=0.0),
                "A_log": WeightSpec((i, n), init="uniform", lo=-1.0, hi=1.5), "D": WeightSpec((i,), init="ones_normal"),
                "o": WeightSpec((self.width, i))}

    def load(self, tensors, ctx: BuildContext) -> None:
        p = self.prefix
        f32 = dict(device=ctx.device, dtype=torch.float32)
        i, n, r = self.inner, self.state_dim, self.dt_rank
        stored = tensors[p + "in"].to(ctx.dtype)
        w = torch.zeros((self.width, self.z_at + pad8(i)), dtype=ctx.dtype)
        w[:, :i] = stored[:i].t()
        w[:, self.z_at:self.z_at + i] = stored[i:].t()
        self.w_in = w.to(ctx.device).contiguous()
        stored = tensors[p + "x"].to(ctx.dtype)                # rows: low | B | C
        w = torch.zeros((i, self.c_at + pad8(n)), dtype=ctx.dtype)
        w[:, :r] = stored[:r].t()
        w[:, self.b_at:self.b_at + n] = stored[r:r + n].t()
        w[:, self.c_at:self.c_at + n] = stored[r + n:].t()
        self.w_x = w.to(ctx.device).contiguous()
        w = torch.zeros((self.b_at, i), dtype=ctx.dtype)       # (the rank's padding meets zeros)
        w[:r] = tensors[p + "dt"].to(ctx.dtype).t()
        self.w_dt = w.to(ctx.device).contiguous()
        self.w_o = tensors[p + "o"].to(device=ctx.device, dtype=ctx.dtype).t().contiguous()
        self.dt_bias = tensors[p + "dt.b"].to(**f32).contiguous()
        self.a_log = tensors[p + "A_log"].to(**f32).contiguous()
        self.skip = tensors[p + "D"].to(**f32).contiguous()

    def forward(self, x, step, binding: LayerBinding, residual=None):
        n, i, s = x.shape[0], self.inner, self.state_dim
        proj = ops.gemm(x, self.w_in)
        xs = self.conv.forward(proj[:, :i], step, binding.state[:, self.state_floats:])
        low = ops.gemm(xs, self.w_x)
        dt = ops.gemm_f32_out(low[:, :self.b_at], self.w_dt)
        out = torch.empty((n, i), dtype=x.dtype, device=x.device)
        ops.selective_scan(xs, dt, self.dt_bias, self.a_log, low[:, self.b_at:self.b_at + s], low[:, self.c_at:self.c_at + s],
                           self.skip, proj[:, self.z_at:self.z_at + i], binding.state, out, step.row_slot, step.row_last,
                           segments=step.plan(segment_plan.planner()))
        return ops.gemm(out, self.w_o, sink=residual)


register_part("mixer", "selective_scan", SelectiveScan)
