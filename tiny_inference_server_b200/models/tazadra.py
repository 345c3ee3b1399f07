"""The Tazadra decoder, put together from parts: token embedding; layers whose sublayers read the stream as it is, with a norm
behind each, ``x += mult * norm1(mixer(x))``, ``x += mult * norm2(ff(x))``; three kinds of mixer (a selective scan; attention in
chunks with bounded scores, over keys and values of its own or of an earlier layer; a time mixer with a matrix state); a
feed-forward of one clamped gated unit or a routed mixture whose weights multiply the experts' inputs; final norm; logits from
a matrix of their own, bounded by a tanh.

Tensor names::

    embed                                   (vocab, width)
    l<i>.norm1, l<i>.norm2                  (width,)    behind the mixer and behind the feed-forward (layers that have one)
    l<i>.mix.*                              the mixer's tensors (``parts.selective_scan.SelectiveScan``,
                                            ``parts.normed_attention.NormedRotaryAttention``, ``parts.time_mix.TimeMix``)
    l<i>.mlp.gate, .up, .down               the dense feed-forward (``parts.feed_forward.SwiGLU`` with the clamped gating)
    l<i>.mlp.e<j>.*, .router                the mixture (``parts.feed_forward.RoutedExperts``)
    final.norm                              (width,)
    head                                    (vocab, width)

Linear weights are stored ``(out, in)``.
"""
from __future__ import annotations

from typing import List

from ..config.model_config import TazadraConfig
from ..kernels import ops
from ..parts.block import Block
from ..parts.embedding import Embedding, LMHead
from ..parts.feed_forward import RoutedExperts, SwiGLU
from ..parts.normed_attention import NormedRotaryAttention
from ..parts.norms import RMSNormMeanEps, StreamAsIs
from ..parts.positions import RotaryBanded
from ..parts.selective_scan import SelectiveScan
from ..parts.stream import ResidualStream
from ..parts.time_mix import TimeMix
from ..registry import register_architecture
from .base import Model, ScheduleEntry, StepOutput


def _feed_forward(cfg: TazadraConfig, i: int, prefix: str):
    f = cfg.layers[i].get("mlp")
    if f is None:
        return None
    if f["kind"] == "dense":
        return SwiGLU(cfg.hidden_size, f["ff"], prefix=prefix, names={"gate": "gate", "up": "up", "down": "down"},
                      stored_out_in=True, form=ops.gate_clamped(f["limit"]))
    # sigmoid scores choose and weigh as they are; a weight multiplies its expert's input
    return RoutedExperts.from_config(cfg, prefix=prefix, layer_index=i, scores="sigmoid", correction=False, renorm=False,
                                     weigh_input=True)


class TazadraModel(Model):
    def __init__(self, cfg: TazadraConfig):
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
            key = (rot["dims"], float(rot["base"]), tuple(sorted((rot.get("scaling") or {}).items())))
            if key not in rotations:
                rotations[key] = RotaryBanded(m["dim"], rot["base"], cfg.max_context, scaling=rot.get("scaling"),
                                              rotary_dim=rot["dims"])
            return rotations[key]

        def mixer(i, prefix):
            kind, m = cfg.layers[i]["type"], cfg.layers[i]["mixer"]
            if kind == "mamba1":
                return SelectiveScan.from_config(cfg, prefix=prefix, layer_index=i)
            if kind == "wkv":
                return TimeMix.from_config(cfg, prefix=prefix, layer_index=i)
            return NormedRotaryAttention.from_config(cfg, prefix=prefix, layer_index=i, position=rotation(m), qk_norm="whole",
                                                     chunked=True, cache_chunks=cfg.cache_chunks(i), softcap=m.get("softcap"),
                                                     head_gate=True)

        def behind(name):
            return RMSNormMeanEps(width, eps, prefix=name, weight_name="", gain=cfg.residual_mult)

        self.embedding = Embedding(cfg.vocab_size, width, weight_name="embed")
        as_is = StreamAsIs(width)
        self.blocks: List[Block] = []
        for i in range(cfg.num_layers):
            p = f"l{i}."
            ffn = _feed_forward(cfg, i, p + "mlp.")
            self.blocks.append(Block(as_is, mixer(i, p + "mix."), as_is if ffn is not None else None, ffn, prefix=p,
                                     post_mixer_norm=behind(p + "norm1"),
                                     post_ffn_norm=behind(p + "norm2") if ffn is not None else None))
        self.final_norm = RMSNormMeanEps(width, eps, prefix="final.norm", weight_name="")
        self.lm_head = LMHead(cfg.vocab_size, width, None, weight_name="head", softcap=cfg.logit_softcap)
        self.entries = [ScheduleEntry(b, source=cfg.layers[i]["mixer"].get("kv_from") if cfg.layers[i]["type"] == "attention" else None)
                        for i, b in enumerate(self.blocks)]

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


def build(cfg: TazadraConfig) -> TazadraModel:
    return TazadraModel(cfg)


register_architecture(TazadraConfig.architecture, TazadraConfig, build)
