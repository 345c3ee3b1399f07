"""A time mixer in the manner of RWKV: a matrix state with a decay per key channel that depends on the token, a bonus for the
current token, and inputs that are mixed with the token before."""
from __future__ import annotations

from typing import Dict

import torch

from ..kernels import ops, segment_plan
from ..registry import register_part
from .base import BuildContext, LayerBinding, Mixer, StateSpec, WeightSpec
from .window_attention import pad8

#: the mixes, in the order of the kernels' operands
MIXES = ("r", "k", "v", "g", "w")


class TimeMix(Mixer):
    """Per head a state ``S`` (``dim x dim``, float32, zero at the start of a sequence).  With ``h'`` the previous token's input
    (zeros for the first token), every s of r, k, v, g, w reads a mix of its own, ``m_s = h + (h' - h) * mu_s``:

    * ``r, k, v = W_s m_s`` (``num_heads`` heads of ``dim``), ``gate = silu(W_g m_g)``;
    * a decay per head and key channel, ``w = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))``;
    * ``o = (S + diag(u) k v^T)^T r`` (the bonus ``u`` reaches the current token only), then ``S <- diag(w) S + k v^T``;
    * every head's ``o`` is divided by its root mean square (``eps`` inside the root); the heads side by side times ``norm``
      (a weight per element of all heads) times the gate; then ``W_o``.

    Tensor names below the prefix: ``r, k, v, g, o, w1, w2`` (stored (out, in)), ``mu.r`` .. ``mu.w``, ``w0``, ``u`` (num_heads,
    dim), ``norm``.  The mixes are formed in 32-bit; the decay, the state, the recurrence and the norm are 32-bit.  The state
    of a request is S of every head followed by its last input."""

    graph_safe = True
    fuses_residual = True

    def __init__(self, width: int, num_heads: int, dim: int, decay_rank: int, eps: float, prefix: str = ""):
        super().__init__(prefix)
        self.width, self.num_heads, self.dim, self.decay_rank, self.eps = width, num_heads, dim, decay_rank, float(eps)
        self.nh = num_heads * dim
        self.state_matrix = num_heads * dim * dim
        self.w_rkvg = self.w_low = self.w_decay = self.w_o = self.mu = self.w_bias = self.bonus = self.norm_w = None

    @classmethod
    def from_config(cls, cfg, prefix: str, layer_index: int, lag: int = 0, position=None):
        m = cfg.layers[layer_index]["mixer"]
        if "decay_rank" not in m:
            raise ValueError(f"layers[{layer_index}].mixer: the rank of the decay's projection is not known "
                             f"(read the configuration with registry.config_from_folder)")
        return cls(cfg.hidden_size, m["heads"], m["dim"], m["decay_rank"], cfg.norm_eps, prefix=prefix)

    def step_planners(self):
        return (segment_plan.planner(),)

    def state_spec(self) -> StateSpec:
        return StateSpec((self.state_matrix + self.width,), torch.float32)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        w, n, r = self.width, self.nh, self.decay_rank
        specs = {"mu." + s: WeightSpec((w,), init="uniform") for s in MIXES}
        specs.update({s: WeightSpec((n, w)) for s in "rkvg"})
        specs.update({"w1": WeightSpec((r, w)), "w2": WeightSpec((n, r)), "w0": WeightSpec((n,), init="uniform", lo=-5.0, hi=0.0),
                      "u": WeightSpec((self.num_heads, self.dim)), "norm": WeightSpec((n,), init="ones_normal"),
                      "o": WeightSpec((w, n))})
        return specs

    def load(self, tensors, ctx: BuildContext) -> None:
        p = self.prefix
        dev = dict(device=ctx.device, dtype=ctx.dtype)
        f32 = dict(device=ctx.device, dtype=torch.float32)
        self.w_rkvg = torch.stack([tensors[p + s].t() for s in "rkvg"]).to(**dev).contiguous()       # (4, width, heads * dim)
        rank = pad8(self.decay_rank)
        low = torch.zeros((self.width, rank), dtype=ctx.dtype)
        low[:, :self.decay_rank] = tensors[p + "w1"].to(ctx.dtype).t()
        self.w_low = low.to(ctx.device).contiguous()
        up = torch.zeros((rank, pad8(self.nh)), dtype=ctx.dtype)
        up[:self.decay_rank, :self.nh] = tensors[p + "w2"].to(ctx.dtype).t()
        self.w_decay = up.to(ctx.device).contiguous()
        self.w_o = tensors[p + "o"].to(**dev).t().contiguous()
        self.mu = torch.stack([tensors[p + "mu." + s] for s in MIXES]).to(**f32).contiguous()
        self.w_bias = tensors[p + "w0"].to(**f32).contiguous()
        self.bonus = tensors[p + "u"].to(**f32).reshape(-1).contiguous()
        self.norm_w = tensors[p + "norm"].to(**f32).contiguous()

    def forward(self, x, step, binding: LayerBinding, residual=None):
        mixes = ops.token_shift(x, self.mu, binding.state[:, self.state_matrix:], step.row_slot, step.row_last)
        rkvg, low = ops.gemm_side_by_side(mixes, self.w_rkvg, self.w_low, act="tanh")
        decay = ops.gemm(low, self.w_decay)
        out = torch.empty((x.shape[0], self.nh), dtype=x.dtype, device=x.device)
        ops.time_mix(rkvg, decay[:, :self.nh], self.bonus, self.w_bias, self.norm_w, self.eps, binding.state, out, step.row_slot,
                     step.row_last, self.num_heads, self.dim, requests=len(step.segments),
                     segments=step.plan(segment_plan.planner()))
        return ops.gemm(out, self.w_o, sink=residual)


register_part("mixer", "time_mix", TimeMix)
