"""The Lomutar decoder, put together from parts: token embedding; layers with one layer norm whose output both sublayers read,
``h = norm1(x)``, ``x += attention(h) + ff(h)``; attention in a window with rotated and normed queries and keys and a keyless
softmax term, over keys and values of its own or of an earlier layer; a feed-forward gated by gelu, or a routed mixture of
clamped gated units beside a shared one; final layer norm; an output matrix of its own.

Tensor names::

    embed                                   (vocab, width)
    l<i>.norm1, l<i>.norm1.b                (width,)          weight and bias
    l<i>.mix.*                              (``parts.normed_attention.NormedRotaryAttention``)
    l<i>.mlp.gate, .up, .down               the dense feed-forward (``parts.feed_forward.SwiGLU`` gated by gelu)
    l<i>.mlp.e<j>.*, .router, .shared.*     the mixture (``parts.feed_forward.RoutedExperts``)
    final.norm, final.norm.b                (width,)
    head                                    (vocab, width)

Linear weights are stored ``(out, in)``.
"""
from __future__ import annotations

from typing import List

from ..config.model_config import LomutarConfig
from ..kernels import ops
from ..parts.block import Block
from ..parts.embedding import Embedding, LMHead
from ..parts.feed_forward import RoutedExperts, SwiGLU
from ..parts.normed_attention import NormedRotaryAttention
from ..parts.norms import LayerNorm
from ..parts.positions import RotaryInterleaved
from ..parts.stream import ResidualStream
from ..registry import register_architecture
from .base import Model, ScheduleEntry, StepOutput


def _feed_forward(cfg: LomutarConfig, i: int, prefix: str):
    f = cfg.layers[i].get("mlp")
    if f is None:
        return None
    if f["kind"] == "dense":
        return SwiGLU(cfg.hidden_size, f["ff"], prefix=prefix, names={"gate": "gate", "up": "up", "down": "down"},
                      stored_out_in=True, form=ops.gate_gelu_tanh())
    # a softmax over all experts scores them, a group is as strong as its best expert, the scores are the weights
    shared = f.get("shared")
    return RoutedExperts.from_config(cfg, prefix=prefix, layer_index=i, scores="softmax", correction=False,
                                     group_score="best", renorm=False, form=ops.gate_clamped(f["expert"]["limit"]),
                                     shared_form=ops.gate_clamped(shared["limit"]) if shared else None, shared_gated=False)


class LomutarModel(Model):
    def __init__(self, cfg: LomutarConfig):
        super().__init__()
        self.config = cfg
        self.vocab_size = cfg.vocab_size
        self.max_positions = cfg.max_context
        width, eps = cfg.hidden_size, cfg.norm_eps
        rotations = {}

        def rotation(m):
            """One table per kind of rotation, whatever number of layers has it."""
            rot = m.get("rot")
            if not rot:
                return None
            key = (rot["dims"], float(rot["base"]), float((rot.get("scaling") or {}).get("factor", 1.0)))
            if key not in rotations:
                rotations[key] = RotaryInterleaved(m["dim"], key[1], cfg.max_context, rotary_dim=key[0], factor=key[2])
            return rotations[key]

        self.embedding = Embedding(cfg.vocab_size, width, weight_name="embed")
        self.blocks: List[Block] = []
        for i, layer in enumerate(cfg.layers):
            p = f"l{i}."
            mixer = NormedRotaryAttention.from_config(cfg, prefix=p + "mix.", layer_index=i, position=rotation(layer["mixer"]),
                                                      cache_window=cfg.cache_window(i))
            self.blocks.append(Block(LayerNorm(width, eps, prefix=p + "norm1", weight_name=""), mixer, None,
                                     _feed_forward(cfg, i, p + "mlp."), prefix=p, parallel=True))
        self.final_norm = LayerNorm(width, eps, prefix="final.norm", weight_name="")
        self.lm_head = LMHead(cfg.vocab_size, width, None, weight_name="head")
        self.entries = [ScheduleEntry(b, source=cfg.layers[i]["mixer"].get("kv_from")) for i, b in enumerate(self.blocks)]

    def top_parts(self):
        return [self.embedding, *self.blocks, self.final_norm, self.lm_head]

    def forward(self, step, want_rows, aux: bool = False) -> StepOutput:
        stream = ResidualStream(self.embedding.forward(step.tokens))
        for e in self.entries:
            e.block.forward(stream, step, e.binding)
        h = stream.normed(self.final_norm)
        if not getattr(step, "want_identity", False):
            h = h.index_select(0, want_rows)
        return StepOutput(main=self.lm_head.forward(h))


def build(cfg: LomutarConfig) -> LomutarModel:
    return LomutarModel(cfg)


register_architecture(LomutarConfig.architecture, LomutarConfig, build)
