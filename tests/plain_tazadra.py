"""Plain, slow implementation of the Tazadra decoder: whole sequences, no cache, one function per mechanism, ordinary
tensor arithmetic in float64.  It takes the configuration as the dictionary of ``config.json`` and the weights as a
dictionary of tensors by name (it reads both on its own) and shares no code with the engine package.

Notation: ``L`` tokens of one sequence, ``t`` a position from 0, ``h`` the input of a sublayer, ``W[name]`` a tensor
stored ``(out, in)``.

* layer: ``x += mult * norm1(mixer(x))``, then ``x += mult * norm2(ff(x))``: norms behind the sublayers only;
* mixers: ``selective_scan_mixer`` (a decay per channel and state), ``attention`` (queries and keys normed as a whole and
  then rotated, bounded scores, chunks, a keyless term, a gate per head, own or shared keys), ``time_mix`` (a matrix state
  with a decay per key channel, a bonus for the current token, inputs mixed with the token before);
* feed-forward: ``clamped_unit``, or ``expert_mixture``: sigmoid scores, the weight on the expert's input.
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


def rms(z, eps: float):
    return torch.sqrt((z * z).mean(-1, keepdim=True) + eps)


def rms_norm(z, w, eps: float):
    return z / rms(z, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(x, w, b):
    """``x`` (L, C), ``w`` (C, taps): the last column weighs the current row, rows before the first are zero."""
    L, taps = x.shape[0], w.shape[1]
    out = b.expand_as(x).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < L:
            out[back:] += w[:, j] * x[:L - back]
    return out


def selective_scan(x, dt, A, B, C, D):
    """``x``, ``dt`` (L, channels), ``A`` (channels, N), ``B``, ``C`` (L, N), ``D`` (channels): channel c's state takes
    ``S_n = exp(dt A_n) S_n + dt x B_n`` and gives ``sum_n S_n C_n + D x``."""
    S = torch.zeros_like(A)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out


def selective_scan_mixer(h, W, p, m, eps):
    inner, rank, N = m["inner"], m["dt_rank"], m["state"]
    x, z = (h @ W[p + "in"].T).split(inner, dim=-1)
    x = silu(causal_conv(x, W[p + "conv"], W[p + "conv.b"]))
    low, B, C = (x @ W[p + "x"].T).split([rank, N, N], dim=-1)
    dt = torch.nn.functional.softplus(low @ W[p + "dt"].T + W[p + "dt.b"], threshold=1e9)
    y = selective_scan(x, dt, -torch.exp(W[p + "A_log"]), B, C, W[p + "D"])
    return (y * silu(z)) @ W[p + "o"].T


def scaled_frequencies(rot: dict):
    """Frequencies of the rotation's pairs; long waves slowed down by ``factor``, short ones kept, those between blended."""
    dims = rot["dims"]
    out = []
    for i in range(dims // 2):
        f = float(rot["base"]) ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_pairs(z, rot, first_position: int = 0):
    """``z`` (L, heads, dim): channel 2i turns with channel 2i + 1 by ``t * f_i``."""
    out = z.clone()
    for i, f in enumerate(scaled_frequencies(rot)):
        ang = torch.arange(first_position, first_position + z.shape[0], dtype=z.dtype)[:, None] * f
        a, b = z[..., 2 * i], z[..., 2 * i + 1]
        out[..., 2 * i] = a * torch.cos(ang) - b * torch.sin(ang)
        out[..., 2 * i + 1] = b * torch.cos(ang) + a * torch.sin(ang)
    return out


def prepared(z, w, heads, dim, rot, eps):
    """Queries or keys as the scores take them: normed over all heads at once, then rotated."""
    z = rms_norm(z, w, eps).view(z.shape[0], heads, dim)
    return rotate_pairs(z, rot) if rot else z


def chunk_softmax(q, k, v, scale, softcap, size, sink):
    """``q`` (L, H, D), ``k`` (L, G, D), ``v`` (L, G, V): row t sees the keys up to t of its own chunk of ``size`` positions
    (None: all); scores bounded by ``softcap`` (None: not); the denominator of head h also holds ``exp(sink_h)``."""
    L, H, _ = q.shape
    G = k.shape[1]
    at = torch.arange(L)
    seen = at[:, None] >= at[None, :]
    if size is not None:
        seen = seen & (at[:, None] // size == at[None, :] // size)
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(~seen, float("-inf"))
        big = torch.maximum(s.max(-1).values, sink[h])
        e = torch.exp(s - big[:, None])
        out[:, h] = (e / (e.sum(-1) + torch.exp(sink[h] - big))[:, None]) @ v[:, g]
    return out


def attention(h, W, p, m, eps, source=None):
    """Returns (output, (keys, values)); ``source``: the keys and values of the layer that this one reads."""
    L, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = prepared(h @ W[p + "q"].T, W[p + "q.norm"], H, D, m.get("rot"), eps)
    if source is None:
        source = (prepared(h @ W[p + "k"].T, W[p + "k.norm"], G, D, m.get("rot"), eps), (h @ W[p + "v"].T).view(L, G, m["vdim"]))
    k, v = source
    o = chunk_softmax(q, k, v, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"), W[p + "sink"])
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(L, -1) @ W[p + "o"].T, source


def time_mix_scan(r, k, v, w, u):
    """``r, k, v, w`` (L, H, D), ``u`` (H, D): ``o_t = (S + diag(u) k v^T)^T r``, then ``S = diag(w) S + k v^T``."""
    L, H, D = r.shape
    S = torch.zeros(H, D, D, dtype=r.dtype)
    out = torch.zeros(L, H, D, dtype=r.dtype)
    for t in range(L):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return out


def time_mix(h, W, p, m, eps):
    L, H, D = h.shape[0], m["heads"], m["dim"]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])

    def mixed(s):
        return h + (before - h) * W[p + "mu." + s]

    r, k, v = ((mixed(s) @ W[p + s].T).view(L, H, D) for s in "rkv")
    gate = silu(mixed("g") @ W[p + "g"].T)
    w = torch.exp(-torch.exp(torch.tanh(mixed("w") @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"])).view(L, H, D)
    o = time_mix_scan(r, k, v, w, W[p + "u"])
    o = (o / rms(o, eps)).reshape(L, H * D) * W[p + "norm"] * gate
    return o @ W[p + "o"].T


def clamped_unit(h, W, p, limit):
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def silu_unit(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, W_router, router):
    """(chosen (L, top), weights (L, top)): the largest sigmoid scores, as they are."""
    s = torch.sigmoid(h @ W_router.T)
    chosen = torch.topk(s, router["top"], dim=-1).indices
    return chosen, s.gather(1, chosen)


def expert_mixture(h, W, p, f):
    chosen, weights = route(h, W[p + "router"], f["router"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        for j in range(f["router"]["top"]):
            rows = (chosen[:, j] == e).nonzero().flatten()
            if len(rows):
                out[rows] += silu_unit(weights[rows, j:j + 1] * h[rows], W, f"{p}e{e}.")
    return out


def feed_forward(h, W, p, f):
    return clamped_unit(h, W, p, f["limit"]) if f["kind"] == "dense" else expert_mixture(h, W, p, f)


def plain_forward(c: dict, W: dict, tokens, return_layers: bool = False):
    eps, mult = c["norm"]["eps"], c.get("residual_mult", 1.0)
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    layers, held = [], {}
    for i, layer in enumerate(c["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            out, held[i] = attention(x, W, p + "mix.", m, eps, held[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            out = {"mamba1": selective_scan_mixer, "wkv": time_mix}[layer["type"]](x, W, p + "mix.", m, eps)
        x = x + mult * rms_norm(out, W[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + mult * rms_norm(feed_forward(x, W, p + "mlp.", layer["mlp"]), W[p + "norm2"], eps)
        layers.append(x.clone())
    logits = rms_norm(x, W["final.norm"], eps) @ W["head"].T
    cap = c.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    if return_layers:
        return logits, torch.stack(layers)
    return logits
