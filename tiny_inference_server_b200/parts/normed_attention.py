"""Grouped-query attention whose queries and keys are rotated and normed, in a window or in chunks, with a keyless term in the
softmax, over keys and values of its own or of an earlier layer."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..kernels import attention_plan, ops, window_plan
from ..registry import register_part
from .base import BuildContext, KVSpec, LayerBinding, Mixer, WeightSpec
from .window_attention import pad8

#: ``cache_window`` of a layer whose keys every reader sees inside its own window
OWN_WINDOW = "own"


class NormedRotaryAttention(Mixer):
    """Causal softmax attention with ``num_heads`` query heads over ``kv_heads`` key/value heads (query head h reads key/value
    head ``h // (num_heads / kv_heads)``):

    * ``q = Wq h``, ``k = Wk h`` (``dim`` elements a head), ``v = Wv h`` (``v_dim``), no biases;
    * ``position`` (a ``RotaryHalf`` family member, None: none) rotates the first ``position.rotary_dim`` elements of every
      query and key head by the token's position;
    * ``qk_norm``: every query and key head is *then* divided by its root mean square over ``dim`` (``eps`` inside the root, no
      weight); or, ``qk_norm`` ``"whole"``, all query heads together, and all key heads together, are divided by their root mean
      square and multiplied by weights ``q.norm`` and ``k.norm`` *before* the rotation; None: no norm;
    * ``score = (q . k) * scale`` over the keys ``p - window + 1 .. p`` (``window`` None: ``0 .. p``), softmax in 32-bit; with
      ``has_sink`` its denominator also holds ``exp(sink[h])``, a term without a key or a value behind it; ``chunked``: a row
      sees the keys up to itself of its own chunk of ``window`` positions instead (chunks are counted from position 0);
      ``softcap`` c (None: none): a score s becomes ``c * tanh(s / c)``;
    * ``head_gate``: head h's output times ``sigmoid(Wg h)_h``, one number a head;
    * ``Wo`` on the heads' outputs side by side.

    How it runs: keys and values of one width that is a multiple of 16 (16..256), at most 64 query heads a kv head: the paged
    attention kernels of the rotary GQA model (tcgen05 tiles for long portions, key splits over a cluster for decode rows,
    which also rotate, norm and store the row's own key, unless heads are normed together, scores bounded or outputs gated);
    any other widths: the kernels of windowed attention.  Where the attention kernel does not, a launch in front of it rotates,
    norms and stores.  The choice depends on the layer's sizes only, so all layers that use a plane
    agree on its row format.

    The cache holds the keys as the scores take them (rotated, normed) and the values.  ``reads_cache``: the layer has no key
    and value projections and stores nothing; its schedule entry names the entry whose plane it reads
    (``models.base.ScheduleEntry.source``), which holds keys and values of the same heads and widths.  A layer whose plane
    is read by layers with wider windows keeps as much as the widest of them sees (``cache_window``), one that layers with chunks
    read (``cache_chunks``, the sizes of all readers' chunks; empty: some reader sees everything) as far back as the furthest
    start of a chunk.

    Tensor names below the prefix: ``q, k, v, o, g`` (stored (out, in)), ``sink``, ``q.norm, k.norm``."""

    graph_safe = True
    fuses_residual = True

    def __init__(self, width: int, num_heads: int, kv_heads: int, dim: int, v_dim: int, scale: float, eps: float, position,
                 window: Optional[int] = None, has_sink: bool = True, qk_norm=True, reads_cache: bool = False,
                 cache_window=OWN_WINDOW, prefix: str = "", chunked: bool = False, cache_chunks=None,
                 softcap: Optional[float] = None, head_gate: bool = False):
        super().__init__(prefix)
        if num_heads % kv_heads:
            raise ValueError(f"{num_heads} query heads are not a multiple of {kv_heads} kv heads")
        self.width, self.num_heads, self.kv_heads, self.dim, self.v_dim = width, num_heads, kv_heads, dim, v_dim
        self.scale, self.eps, self.position, self.window = float(scale), float(eps), position, window
        self.has_sink, self.qk_norm, self.reads_cache = has_sink, bool(qk_norm) and qk_norm != "whole", reads_cache
        self.whole_norm = qk_norm == "whole"
        self.chunked, self.softcap, self.head_gate = chunked, (float(softcap) if softcap else None), head_gate
        self.cache_chunks = ()
        if chunked:
            self.cache_chunks = tuple(sorted(set(cache_chunks))) if cache_chunks is not None else ((window,) if window else ())
            cache_window = None
            if self.cache_chunks and window not in self.cache_chunks:
                raise ValueError(f"chunks of {window} keys over a plane that keeps chunks of {self.cache_chunks}")
        self.cache_window = window if cache_window == OWN_WINDOW else cache_window
        if self.cache_window is not None and (window is None or window > self.cache_window):
            raise ValueError(f"a window of {window} keys over a plane that keeps {self.cache_window}")
        self.paged = (dim == v_dim and dim % 16 == 0 and 16 <= dim <= 256 and num_heads // kv_heads <= 64 and self.scale > 0)
        self.nq, self.nk, self.nv, self.no = num_heads * dim, kv_heads * dim, kv_heads * v_dim, num_heads * v_dim
        self.gate_at = pad8(self.nq if reads_cache else self.nq + self.nk + self.nv)
        self.w_in = self.w_o = self.sink = self.qk_weight = None

    @classmethod
    def from_config(cls, cfg, prefix: str, layer_index: int, lag: int = 0, position=None, cache_window=OWN_WINDOW, **options):
        m = cfg.layers[layer_index]["mixer"]
        mask = m.get("mask")
        return cls(cfg.hidden_size, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], cfg.norm_eps, position,
                   window=mask["size"] if mask else None, reads_cache=m.get("kv_from") is not None,
                   cache_window=cache_window, prefix=prefix, **options)

    def children(self):
        return (self.position,) if self.position is not None else ()

    def kv_spec(self) -> KVSpec:
        return KVSpec(self.kv_heads, self.dim, self.cache_window, 0, k_dim=self.dim, v_dim=self.v_dim, chunks=self.cache_chunks)

    def step_planners(self):
        plan = attention_plan if self.paged else window_plan
        return (plan.planner(self.num_heads // self.kv_heads),)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        specs = {"q": WeightSpec((self.nq, self.width))}
        if not self.reads_cache:
            specs.update({"k": WeightSpec((self.nk, self.width)), "v": WeightSpec((self.nv, self.width))})
        specs["o"] = WeightSpec((self.width, self.no))
        if self.has_sink:
            specs["sink"] = WeightSpec((self.num_heads,), init="uniform", lo=-1.0, hi=1.0)
        if self.whole_norm:
            specs["q.norm"] = WeightSpec((self.nq,), init="ones_normal")
            if not self.reads_cache:
                specs["k.norm"] = WeightSpec((self.nk,), init="ones_normal")
        if self.head_gate:
            specs["g"] = WeightSpec((self.num_heads, self.width))
        return specs

    def load(self, tensors, ctx: BuildContext) -> None:
        p = self.prefix
        names = ("q",) if self.reads_cache else ("q", "k", "v")
        w = torch.cat([tensors[p + n] for n in names], dim=0).to(ctx.dtype)
        cols = w.shape[0]
        total = self.gate_at + pad8(self.num_heads) if self.head_gate else pad8(cols)
        w_in = torch.zeros((self.width, total), dtype=ctx.dtype)             # rows of the product start on 16-byte boundaries
        w_in[:, :cols] = w.t()
        if self.head_gate:
            w_in[:, self.gate_at:self.gate_at + self.num_heads] = tensors[p + "g"].to(ctx.dtype).t()
        if self.whole_norm:
            norms = [tensors[p + n + ".norm"] for n in (("q",) if self.reads_cache else ("q", "k"))]
            self.qk_weight = torch.cat(norms).to(device=ctx.device, dtype=torch.float32).contiguous()
        self.w_in = w_in.to(ctx.device).contiguous()
        self.w_o = tensors[p + "o"].to(device=ctx.device, dtype=ctx.dtype).t().contiguous()
        if self.has_sink:
            self.sink = tensors[p + "sink"].to(device=ctx.device, dtype=torch.float32).contiguous()

    def forward(self, x, step, binding: LayerBinding, residual=None):
        n = x.shape[0]
        g = binding.kv_group
        table, page_size = step.block_tables[g], step.page_sizes[g]
        proj = ops.gemm(x, self.w_in)
        pos = self.position
        cos, sin, interleaved = (pos.cos, pos.sin, pos.interleaved) if pos is not None else (None, None, True)
        out = torch.empty((n, self.no), dtype=x.dtype, device=x.device)
        gate = proj[:, self.gate_at:self.gate_at + self.num_heads] if self.head_gate else None
        in_kernel = self.paged and interleaved and not self.whole_norm and not self.softcap and not self.chunked and gate is None and ops.rotary_fusable(proj, step, self.num_heads, self.kv_heads, self.dim, pairs=True)
        if not in_kernel:
            ops.rotate_norm_store(proj, self.num_heads, 0 if self.reads_cache else self.kv_heads, self.dim, self.v_dim, cos, sin,
                                  interleaved, self.qk_norm, self.eps, binding.k_pages, binding.v_pages, table, step.positions,
                                  step.row_slot, page_size, step.fault, permuted=self.paged, whole_weight=self.qk_weight)
        if self.paged:
            rotary = ops.PairRotary(cos, sin, self.eps if self.qk_norm else None) if in_kernel else None
            ops.paged_attention(proj, out, binding.kv_plane, table, step.positions, step.row_slot, self.num_heads, self.kv_heads,
                                self.dim, page_size, self.window, step.fault, step, rotary=rotary,
                                write_kv=not self.reads_cache, scale=self.scale, sink=self.sink, chunked=self.chunked,
                                softcap=self.softcap, gate=gate)
        else:
            ops.window_attention(proj[:, :self.nq], gate, out, binding.k_pages, binding.v_pages, table, step.positions,
                                 step.row_slot, self.num_heads, page_size, self.window, self.scale, None, None, step.fault,
                                 step, sink=self.sink, gate_per_head=gate is not None, chunked=self.chunked, softcap=self.softcap)
        return ops.gemm(out, self.w_o, sink=residual)


register_part("mixer", "normed_rotary_attention", NormedRotaryAttention)
