"""Plain, slow implementation of the Lomutar decoder: whole sequences, no cache, one function per mechanism, ordinary
tensor arithmetic in float64.  It takes the configuration as the dictionary of ``config.json`` and the weights as a
dictionary of tensors by name (it reads both on its own) and shares no code with the engine package.

Notation: ``L`` tokens of one sequence, ``t`` a position from 0, ``h`` the input of a sublayer, ``W[name]`` a tensor
stored ``(out, in)``.

* layer: ``h = layer_norm(x)``, ``x += attention(h) + ff(h)``: one norm, both sublayers read its output;
* attention: queries and keys rotated (neighbouring channels paired, frequencies over a constant), then divided by their
  root mean square per head; a window; a keyless term in the softmax; a layer may read an earlier layer's keys and values;
* feed-forward: ``gelu_gated_ff``, or ``expert_mixture``: a softmax over all experts, the best groups, the best experts in
  them, clamped gated units, and a unit that every token passes.
"""
from __future__ import annotations

import json
import math
import os

import torch

F64 = torch.float64


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def read_weights(folder: str, dtype=F64) -> dict:
    from safetensors.torch import load_file
    return {k: v.to(dtype) for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}


def layer_norm(z, w, b, eps: float):
    mean = z.mean(-1, keepdim=True)
    centred = z - mean
    var = (centred * centred).mean(-1, keepdim=True)
    return centred / torch.sqrt(var + eps) * w + b


def unit_rms(z, eps: float):
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps)


def rotate_pairs(z, rot, first_position: int = 0):
    """``z`` (L, heads, dim): of the first ``rot.dims`` channels of each head, channel 2i turns with channel 2i + 1 by
    ``t * base^(-2i/dims) / factor``."""
    dims = rot["dims"]
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    out = z.clone()
    for i in range(dims // 2):
        f = float(rot["base"]) ** (-2.0 * i / dims) / factor
        ang = torch.arange(first_position, first_position + z.shape[0], dtype=z.dtype)[:, None] * f
        a, b = z[..., 2 * i], z[..., 2 * i + 1]
        out[..., 2 * i] = a * torch.cos(ang) - b * torch.sin(ang)
        out[..., 2 * i + 1] = b * torch.cos(ang) + a * torch.sin(ang)
    return out


def prepared(z, heads, dim, rot, eps):
    """Queries or keys as the scores take them: rotated, then normed per head."""
    z = z.view(z.shape[0], heads, dim)
    if rot:
        z = rotate_pairs(z, rot)
    return unit_rms(z, eps)


def window_softmax(q, k, v, scale, size, sink):
    """``q`` (L, H, D), ``k`` (L, G, D), ``v`` (L, G, V): row t sees keys ``t - size + 1 .. t`` (size None: 0 .. t); the
    denominator of head h also holds ``exp(sink_h)``."""
    L, H, _ = q.shape
    G = k.shape[1]
    dist = torch.arange(L)[:, None] - torch.arange(L)[None, :]
    seen = dist >= 0
    if size is not None:
        seen = seen & (dist < size)
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, float("-inf"))
        big = torch.maximum(s.max(-1).values, sink[h])
        e = torch.exp(s - big[:, None])
        out[:, h] = (e / (e.sum(-1) + torch.exp(sink[h] - big))[:, None]) @ v[:, g]
    return out


def attention(h, W, p, m, eps, source=None):
    """Returns (output, (keys, values)); ``source``: the keys and values of the layer that this one reads."""
    L, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = prepared(h @ W[p + "q"].T, H, D, m.get("rot"), eps)
    if source is None:
        source = (prepared(h @ W[p + "k"].T, G, D, m.get("rot"), eps), (h @ W[p + "v"].T).view(L, G, m["vdim"]))
    k, v = source
    o = window_softmax(q, k, v, m["scale"], (m.get("mask") or {}).get("size"), W[p + "sink"])
    return o.reshape(L, -1) @ W[p + "o"].T, source


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_gated_ff(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def clamped_unit(h, W, p, limit):
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def route(h, W_router, router):
    """(chosen (L, top), weights (L, top)): the best ``top`` experts among those of the best groups; the weights are their
    shares of the softmax over all experts."""
    s = torch.softmax(h @ W_router.T, dim=-1)
    masked = s.clone()
    gr = router.get("groups")
    if gr:
        per = router["experts"] // gr["count"]
        best = s.view(-1, gr["count"], per).max(-1).values
        keep = torch.topk(best, gr["keep"], dim=-1).indices
        allowed = torch.zeros_like(best, dtype=torch.bool).scatter_(1, keep, True)
        masked = s.masked_fill(~allowed.repeat_interleave(per, dim=1), -1.0)
    chosen = torch.topk(masked, router["top"], dim=-1).indices
    return chosen, s.gather(1, chosen)


def expert_mixture(h, W, p, f):
    chosen, weights = route(h, W[p + "router"], f["router"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        for j in range(f["router"]["top"]):
            rows = (chosen[:, j] == e).nonzero().flatten()
            if len(rows):
                out[rows] += weights[rows, j:j + 1] * clamped_unit(h[rows], W, f"{p}e{e}.", f["expert"]["limit"])
    if f.get("shared"):
        out = out + clamped_unit(h, W, p + "shared.", f["shared"]["limit"])
    return out


def feed_forward(h, W, p, f):
    return gelu_gated_ff(h, W, p) if f["kind"] == "dense" else expert_mixture(h, W, p, f)


def plain_forward(c: dict, W: dict, tokens, return_layers: bool = False):
    eps = c["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    layers, held = [], {}
    for i, layer in enumerate(c["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps)
        delta, held[i] = attention(h, W, p + "mix.", m, eps, held[m["kv_from"]] if m.get("kv_from") is not None else None)
        if layer.get("mlp"):
            delta = delta + feed_forward(h, W, p + "mlp.", layer["mlp"])
        x = x + delta
        layers.append(x.clone())
    logits = layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].T
    if return_layers:
        return logits, torch.stack(layers)
    return logits
