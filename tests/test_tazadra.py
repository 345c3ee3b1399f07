"""The Tazadra architecture through the engine against the plain implementation (``plain_tazadra``): configuration and weights,
every mechanism alone with planted inputs, replays cut in every way, configurations drawn at random, slots and pages used
again, long decoding, generation through the scheduler and the command line."""
from __future__ import annotations

import json
import math
import os

import numpy as np
import pytest
import torch

import plain_tazadra as plain
import trace_tools
from tiny_inference_server_b200 import ConfigError, build_model, config_from_dict, config_from_folder
from tiny_inference_server_b200.api import Engine, SamplingParams
from tiny_inference_server_b200.cache.manager import CacheManager
from tiny_inference_server_b200.config import EngineConfig, TazadraConfig
from tiny_inference_server_b200.parts.base import BuildContext, KVSpec, LayerBinding
from tiny_inference_server_b200.trace import TraceReplayer, make_runner
from tiny_inference_server_b200.weights.loader import WeightError

gpu = pytest.mark.gpu


def _scan(inner, state, rank, conv):
    return "mamba1", {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}


def _mix(heads, dim):
    return "wkv", {"heads": heads, "dim": dim}


def _attn(heads, kv, dim, vdim, size, rot=None, scaling=None, base=10000.0, scale=None, softcap=12.0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.5 * dim ** -0.5}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if softcap:
        m["softcap"] = softcap
    if size:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _cfg(vocab, width, layers, eps=1e-5, mult=0.8, cap=9.0):
    c = dict(architecture="Tazadra", vocab=vocab, width=width, norm={"eps": eps}, residual_mult=mult,
             layers=[{"type": k, "mixer": m, "mlp": f} for (k, m), f in layers])
    if cap:
        c["logit_softcap"] = cap
    return c


# readers with larger and with smaller chunks than the layer they read; every kind of mixer and of feed-forward
M1 = _cfg(97, 64, [
    (_mix(2, 16), _dense(96, 0.9)),
    (_attn(4, 2, 16, 16, 13, rot=16, scaling=(4.0, 1.0, 4.0, 64)), _moe(32, 6, 2)),
    (_scan(80, 8, 5, 4), _moe(48, 4, 3)),
    (_attn(4, 2, 16, 16, 30, rot=16, scaling=(4.0, 1.0, 4.0, 64), kv_from=1, softcap=5.0), _dense(64, 1.7)),
    (_attn(4, 2, 16, 16, 5, rot=16, scaling=(4.0, 1.0, 4.0, 64), kv_from=1), None),
])
# sizes that fit no vector or tile; keys and values of different widths; every head with keys of its own; no bound on scores or
# logits; no rotation; a layer that sees everything, read by one with chunks; one expert; a convolution of one tap
M2 = _cfg(53, 40, [
    (_attn(3, 3, 10, 6, 7, rot=4, softcap=None), None),
    (_scan(27, 5, 3, 2), _moe(18, 5, 1)),
    (_attn(2, 1, 6, 14, None), _dense(50, 0.5)),
    (_mix(3, 10), _moe(20, 1, 1)),
    (_attn(2, 1, 6, 14, 11, kv_from=2, scale=0.3), _dense(33, 2.5)),
    (_scan(40, 1, 9, 1), None),
], eps=1e-3, mult=1.0, cap=None)
# widths of the tensor-core kernels: heads of 64 (tcgen05 tiles for long portions), unequal widths, recurrences split over CTAs
M3 = _cfg(200, 128, [
    (_scan(256, 16, 8, 4), _moe(64, 8, 3)),
    (_attn(8, 1, 64, 64, 70, rot=64, scaling=(8.0, 1.0, 4.0, 512), base=5e5), _dense(256, 0.7)),
    (_mix(2, 64), _moe(64, 4, 2)),
    (_attn(4, 2, 32, 48, 33, rot=16), _dense(64, 1.1)),
    (_attn(8, 1, 64, 64, 150, rot=64, scaling=(8.0, 1.0, 4.0, 512), base=5e5, kv_from=1), _moe(128, 4, 4)),
], mult=0.6)
# more query heads a kv head than a decode tile packs; heads of 128; more states than a lane row of 32 holds; wide time mixers
M4 = _cfg(64, 48, [
    (_attn(20, 1, 16, 16, 25, rot=6, base=100.0), _moe(16, 6, 2)),
    (_mix(1, 128), _dense(32, 1.0)),
    (_scan(64, 40, 16, 3), _moe(32, 3, 3)),
    (_attn(2, 2, 128, 128, 41, rot=128, scaling=(2.0, 0.5, 8.0, 100)), None),
    (_mix(3, 24), _dense(24, 0.6)),
], mult=1.3, cap=4.0)

CONFIGS = {"M1": (M1, 16), "M2": (M2, 8), "M3": (M3, 16), "M4": (M4, 4)}
LENGTHS = {"M1": [1, 2, 3, 30, 75, 41, 9, 60], "M2": [1, 5, 40, 33, 17, 64], "M3": [2, 4, 50, 240, 23, 37],
           "M4": [1, 2, 2, 19, 33, 6, 80]}
RANKS = {"M1": 6, "M2": 5, "M3": 16, "M4": 8}


def _raw_with_ranks(raw, rank):
    """The configuration with the ranks of the decays' projections written in (config.json leaves them to the tensors)."""
    raw = json.loads(json.dumps(raw))
    for layer in raw["layers"]:
        if layer["type"] == "wkv":
            layer["mixer"]["decay_rank"] = rank
    return raw


def make_tensors(cfg, seed):
    """Weights of a size that makes every mechanism matter, rounded to bfloat16 so that both precisions and the plain
    implementation hold the same numbers: states that remember hundreds of tokens beside ones that forget at once, gates that
    reach their limits, routers whose logits lie apart, sinks that take a good part of a short chunk, scores near the bound."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, spec in build_model(cfg).expected_tensors().items():
        shape = tuple(spec.shape)
        leaf = name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name
        rnd, uni = torch.randn(shape, generator=gen), torch.rand(shape, generator=gen)
        if name == "embed":
            t = rnd
        elif leaf.endswith("norm") or leaf in ("norm1", "norm2", "final.norm"):
            t = 1.0 + rnd * 0.2
        elif leaf == "mix.sink":
            t = rnd + 1.0
        elif leaf.startswith("mix.mu."):
            t = uni * 1.2 - 0.1
        elif leaf == "mix.w0":
            t = uni * 8.0 - 7.0                       # decays from exp(-e) to exp(-0.001)
        elif leaf == "mix.A_log":
            t = uni * 6.0 - 4.5
        elif leaf == "mix.dt.b":
            t = uni * 3.0 - 2.5
        elif leaf in ("mix.D", "mix.u", "mix.conv.b"):
            t = rnd * 0.7
        elif leaf == "mix.conv":
            t = rnd / math.sqrt(shape[1])
        elif len(shape) == 2:
            t = rnd * {"mlp.router": 2.0}.get(leaf, 1.0) / math.sqrt(shape[1])
        else:
            raise AssertionError(f"no rule for {name} {shape}")
        out[name] = t.to(torch.bfloat16).contiguous()
    return out


def make_folder(raw, seed, folder, rank=8):
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(raw, f)
    save_file(make_tensors(config_from_dict(_raw_with_ranks(raw, rank)), seed), os.path.join(folder, "model.safetensors"))
    return folder


_cache = {}


def all_chosen(raw):
    """The configuration with routers that choose every expert.  A choice that hangs on a rounding replaces an expert by another
    one, and behind the norm of its sublayer, and in the states of the layers above, that stays visible for many tokens: whole
    models in bfloat16 are compared without choices.  The choice itself is compared in float32, and alone."""
    raw = json.loads(json.dumps(raw))
    for layer in raw["layers"]:
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return raw


def _setup(name, tmp_path_factory, dtype="float32"):
    key = name, dtype
    if key not in _cache:
        raw, page = CONFIGS[name]
        if dtype == "bfloat16":
            raw = all_chosen(raw)
        folder = make_folder(raw, 29 + ord(name[-1]), str(tmp_path_factory.mktemp(f"tazadra{name}")), RANKS[name])
        c, W = plain.read_config(folder), plain.read_weights(folder)
        g = torch.Generator().manual_seed(5)
        seqs = {f"r{i}": torch.randint(0, raw["vocab"], (n,), generator=g).tolist() for i, n in enumerate(LENGTHS[name])}
        ref = {rid: plain.plain_forward(c, W, toks).numpy() for rid, toks in seqs.items()}
        _cache[key] = (raw, page, folder, seqs, ref, c, W)
    return _cache[key]


def rel_err(got, ref):
    """Difference of two rows of logits, mean taken off, root mean square, over that of the reference."""
    d = np.asarray(got, dtype=np.float64) - ref
    d = d - d.mean()
    r = ref - ref.mean()
    return float(np.sqrt((d * d).mean()) / max(np.sqrt((r * r).mean()), 1e-9))


#: (in float32 most positions agree to 1e-6; early tokens whose head outputs nearly cancel before the norm, to 2e-4)
TOL = {"float32": 3e-4, "bfloat16": 0.1}
#: The share of positions that may differ by more than the tolerance, and by how much at most: in float32 a router whose scores
#: at the edge of its choice lie within a rounding of each other; in bfloat16 positions whose scores or decays are steep, or
#: whose head reads next to nothing of its state before the norm blows it up (a first token whose bonus nearly cancels).
OUTLIERS = {"float32": 0.01, "bfloat16": 0.06}
OUTLIER_CAP = {"float32": 1.0, "bfloat16": 0.9}


def _steps(mode, seqs, max_live=4):
    if mode == "whole":
        return trace_tools.trace_whole(seqs)
    if mode == "tail":
        return trace_tools.trace_tail(seqs, tail=32)
    if mode == "chunks":
        return trace_tools.trace_chunks(seqs)
    return trace_tools.trace_mixed(seqs, max_live=max_live)


def _replay_and_compare(raw, page, folder, seqs, ref, steps, out_dir, dtype, device, tol, max_live=4, poison=False,
                        shuffle=False, outliers=0.0, cap=1.0):
    """``outliers``: the share of positions that may exceed the tolerance (none of them by more than ``cap``)."""
    runner = make_runner(folder, dtype, trace_tools.max_live_tokens(steps, round_to=64), page_size=page, device=device,
                         max_live=max_live, debug_poison=poison)
    if shuffle:
        import random
        for g in runner.cache.groups:
            g.pool.shuffle(random.Random(3))
    TraceReplayer(runner, out_dir).run(json.dumps(s) for s in steps)
    runner.cache.check()
    assert runner.cache.drained(), "pages or slots were not given back"
    got = trace_tools.gather(steps, out_dir, raw["vocab"])
    over, total = [], sum(len(t) for t in seqs.values())
    for rid, toks in seqs.items():
        for p in range(len(toks)):
            e = rel_err(got[rid][p], ref[rid][p])
            if e >= tol:
                over.append((rid, p, e))
                assert e < cap and len(over) <= outliers * total, \
                    f"logits of {rid} at position {p}: relative error {e} (over the tolerance so far: {over})"
    return runner


# ------------------------------------------------------------------------------------------------
# configuration and weights (CPU)
# ------------------------------------------------------------------------------------------------

def test_config_round_trip_tensor_names_and_shared_planes(tmp_path):
    cfg = config_from_folder(make_folder(M1, 1, str(tmp_path / "m"), 6))
    assert isinstance(cfg, TazadraConfig)
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    assert cfg.layers[0]["mixer"]["decay_rank"] == 6 and cfg.residual_mult == 0.8 and cfg.logit_softcap == 9.0
    model = build_model(cfg)
    names = set(model.expected_tensors())
    assert {"embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.mu.w", "l0.mix.w1", "l0.mix.u", "l1.mix.q.norm", "l1.mix.k.norm",
            "l1.mix.sink", "l1.mix.g", "l1.mlp.e5.gate", "l1.mlp.router", "l2.mix.A_log", "l2.mix.conv.b", "l2.mix.dt.b", "l2.mix.x",
            "l3.mix.q.norm", "l3.mlp.up"} <= names
    assert not any(n.startswith(("l3.mix.k", "l3.mix.v", "l4.mix.k", "l4.norm2", "l4.mlp")) or ".mlp.correction" in n or
                   n.startswith("l0.mlp.gate.b") for n in names)
    # a plane keeps the chunks of all its readers
    specs = model.kv_specs()
    assert [s.chunks if s is not None else None for s in specs] == [None, (5, 13, 30), None, None, None]
    assert model.entries[3].source == 1 and model.entries[4].source == 1 and model.entries[0].source is None
    assert len({id(b.mixer.position) for b in model.blocks if hasattr(b.mixer, "position")}) == 1      # one table a rotation
    open_ended = build_model(config_from_dict(_raw_with_ranks(M2, 5)))
    assert [s.chunks if s is not None else None for s in open_ended.kv_specs()] == [(7,), None, (), None, None, None]
    assert config_from_dict(_raw_with_ranks(M2, 5)).logit_softcap is None


def test_config_errors_name_the_problem():
    def broken(change):
        raw = _raw_with_ranks(M1, 6)
        change(raw)
        with pytest.raises(ConfigError) as e:
            config_from_dict(raw)
        return str(e.value)

    def mixer(i):
        return lambda r: r["layers"][i]["mixer"]

    assert "layers[0].type" in broken(lambda r: r["layers"][0].update(type="gla"))
    assert "layers[0].mixer: dim" in broken(lambda r: mixer(0)(r).pop("dim"))
    assert "dt_rank" in broken(lambda r: mixer(2)(r).update(dt_rank=0))
    assert "conv" in broken(lambda r: mixer(2)(r).update(conv=17))
    assert "state" in broken(lambda r: mixer(2)(r).update(state=300))
    assert "kv heads" in broken(lambda r: mixer(1)(r).update(kv_heads=3))
    assert "scale" in broken(lambda r: mixer(1)(r).pop("scale"))
    assert "softcap" in broken(lambda r: mixer(1)(r).update(softcap=-1.0))
    assert "mask.size" in broken(lambda r: mixer(1)(r)["mask"].update(size=0))
    assert "rot.dims" in broken(lambda r: mixer(1)(r)["rot"].update(dims=18))
    assert "scaling lacks low, original" in broken(lambda r: mixer(1)(r)["rot"].update(scaling={"factor": 2.0, "high": 4.0}))
    assert "kv_from" in broken(lambda r: mixer(3)(r).update(kv_from=3))
    assert "no keys and values of its own" in broken(lambda r: mixer(4)(r).update(kv_from=3))
    assert "no keys and values of its own" in broken(lambda r: mixer(4)(r).update(kv_from=0))
    assert "differ" in broken(lambda r: mixer(3)(r).update(dim=32))
    assert "exceeds" in broken(lambda r: r["layers"][1]["mlp"]["router"].update(top=7))
    assert "limit" in broken(lambda r: r["layers"][0]["mlp"].pop("limit"))
    assert "expert.ff" in broken(lambda r: r["layers"][1]["mlp"]["expert"].update(ff=0))
    assert "mlp.kind" in broken(lambda r: r["layers"][1]["mlp"].update(kind="sparse"))
    assert "residual_mult" in broken(lambda r: r.update(residual_mult="half"))
    assert "logit_softcap" in broken(lambda r: r.update(logit_softcap=0))
    assert "missing keys: width" in broken(lambda r: r.pop("width"))


def test_a_missing_or_misshapen_tensor_is_named(tmp_path):
    from safetensors.torch import load_file, save_file
    from tiny_inference_server_b200.weights.loader import load_weights
    folder = make_folder(M1, 2, str(tmp_path / "m"), 6)
    path = os.path.join(folder, "model.safetensors")
    tensors = load_file(path)
    del tensors["l2.mix.dt.b"]
    tensors["l1.mix.sink"] = torch.zeros(3, dtype=torch.bfloat16)
    tensors["l3.mix.k"] = torch.zeros(32, 64, dtype=torch.bfloat16)        # a layer that reads another's keys has none
    save_file(tensors, path)
    with pytest.raises(WeightError) as e:
        load_weights(folder, build_model(config_from_folder(folder)).expected_tensors())
    assert all(n in str(e.value) for n in ("l2.mix.dt.b", "l1.mix.sink", "l3.mix.k"))
    del tensors["l0.mix.w1"]
    save_file(tensors, path)
    with pytest.raises(ConfigError) as e:
        config_from_folder(folder)
    assert "l0.mix.w1" in str(e.value)


# ------------------------------------------------------------------------------------------------
# the plain implementation against other ways of writing the same sums (CPU)
# ------------------------------------------------------------------------------------------------

def test_plain_mechanisms_written_another_way():
    g = torch.Generator().manual_seed(3)

    def rand(*s):
        return torch.randn(*s, generator=g, dtype=torch.float64)

    # the convolution, tap by tap
    x, w, b = rand(6, 3), rand(3, 4), rand(3)
    got = plain.causal_conv(x, w, b)
    for t in range(6):
        want = b + sum(w[:, 3 - back] * x[t - back] for back in range(4) if t >= back)
        assert torch.allclose(got[t], want)
    # the scan as an explicit sum over the past
    L, C, N = 7, 3, 4
    x, dt, A, B, Cm, D = rand(L, C), torch.rand(L, C, generator=g, dtype=torch.float64), -torch.rand(C, N, generator=g, dtype=torch.float64), \
        rand(L, N), rand(L, N), rand(C)
    got = plain.selective_scan(x, dt, A, B, Cm, D)
    for t in range(L):
        for c in range(C):
            y = D[c] * x[t, c]
            for j in range(t + 1):
                y = y + (Cm[t] * torch.exp(A[c] * dt[j + 1:t + 1, c].sum()) * dt[j, c] * x[j, c] * B[j]).sum()
            assert torch.allclose(got[t, c], y)
    # the time mixer's recurrence as an explicit sum: the current token by the bonus, older ones by the decays between
    L, H, Dm = 6, 2, 3
    r, k, v, u = rand(L, H, Dm), rand(L, H, Dm), rand(L, H, Dm), rand(H, Dm)
    w = torch.rand(L, H, Dm, generator=g, dtype=torch.float64)
    got = plain.time_mix_scan(r, k, v, w, u)
    for t in range(L):
        for h in range(H):
            o = (r[t, h] * u[h] * k[t, h]).sum() * v[t, h]
            for j in range(t):
                o = o + (r[t, h] * torch.prod(w[j + 1:t, h], dim=0) * k[j, h]).sum() * v[j, h]
            assert torch.allclose(got[t, h], o)
    # the rotation: scores depend on the distance only; frequencies in three bands
    rot = {"base": 300.0, "dims": 8, "scaling": {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 100}}
    q = rand(4, 1, 10)
    a, c = plain.rotate_pairs(q, rot, 5), plain.rotate_pairs(q, rot, 11)
    assert abs(float((a[0] * a[2]).sum() - (c[0] * c[2]).sum())) < 1e-9
    assert torch.equal(a[..., 8:], q[..., 8:])
    base = [300.0 ** (-i / 4) for i in range(4)]
    f = plain.scaled_frequencies(rot)
    assert f[0] == base[0] and abs(f[3] - base[3] / 3) < 1e-15 and base[1] / 3 < f[1] < base[1]
    # the softmax, key by key
    L, H, G, D, V, size, cap = 9, 4, 2, 5, 3, 4, 1.5
    qq, kk, vv, sink = rand(L, H, D), rand(L, G, D), rand(L, G, V), rand(H)
    got = plain.chunk_softmax(qq, kk, vv, 0.7, cap, size, sink)
    for t in range(L):
        for h in range(H):
            den, num = math.exp(float(sink[h])), torch.zeros(V, dtype=torch.float64)
            for j in range(t - t % size, t + 1):
                e = math.exp(cap * math.tanh(0.7 * float(qq[t, h] @ kk[j, h // 2]) / cap))
                den += e
                num += e * vv[j, h // 2]
            assert torch.allclose(got[t, h], num / den)
    # the mixture, expert by expert: the weight inside the unit is not the weight outside it
    f = _moe(5, 3, 2)
    W = {f"e{e}.{n}": rand(*((4, 5) if n == "down" else (5, 4))) for e in range(3) for n in ("gate", "up", "down")}
    W["router"] = rand(3, 4)
    h = rand(6, 4)
    got = plain.expert_mixture(h, W, "", f)
    for t in range(6):
        s = torch.sigmoid(W["router"] @ h[t])
        y = torch.zeros(4, dtype=torch.float64)
        for e in sorted(range(3), key=lambda i: -float(s[i]))[:2]:
            z = s[e] * h[t]
            gate = W[f"e{e}.gate"] @ z
            y = y + W[f"e{e}.down"] @ (gate / (1 + torch.exp(-gate)) * (W[f"e{e}.up"] @ z))
        assert torch.allclose(got[t], y)


def test_rotation_tables_in_three_bands():
    from tiny_inference_server_b200.parts.positions import RotaryBanded
    for scaling in (None, {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 300}, {"factor": 2.0, "low": 0.5, "high": 16.0, "original": 5000}):
        rot = {"base": 2000.0, "dims": 24}
        if scaling:
            rot["scaling"] = scaling
        pos = RotaryBanded(32, 2000.0, 700, scaling=scaling, rotary_dim=24)
        want = torch.tensor(plain.scaled_frequencies(rot), dtype=torch.float64)
        assert torch.allclose(pos.frequencies(), want, rtol=1e-12)
        cos, sin = pos.tables()
        ang = torch.arange(700, dtype=torch.float64)[:, None] * want
        assert (cos.double() - torch.cos(ang)).abs().max() < 1e-6 and (sin.double() - torch.sin(ang)).abs().max() < 1e-6


def test_pages_of_finished_chunks_are_given_back():
    """A group that keeps chunks: pages before the earliest start of a reader's chunk leave, no page inside one does."""
    for chunks, page in (((13,), 4), ((5, 13), 4), ((16,), 16), ((7, 30), 8)):
        spec = KVSpec(1, 16, chunks=chunks)
        cache = CacheManager([spec], {}, page_size=page, num_pages=64, max_slots=2, max_positions=200, dtype=torch.float32, device="cpu")
        grp, slot = cache.groups[0], cache.admit()
        at = 0
        for n in (3, 1, 9, 20, 1, 1, 1, 17, 2, 40, 1, 1, 1):
            start = cache.extend(slot, n)
            assert start == at
            first = min(start - start % c for c in chunks)
            assert grp.first[slot] == first // page, (chunks, page, start)
            at += n
            cache.check()
        cache.release(slot)
        assert cache.drained()
    # a smaller pool than the sequence: pages are used again
    cache = CacheManager([KVSpec(1, 16, chunks=(12,))], {}, page_size=4, num_pages=5, max_slots=1, max_positions=200,
                         dtype=torch.float32, device="cpu")
    slot = cache.admit()
    for _ in range(60):
        assert cache.pages_needed(slot, 1) <= cache.free_pages() + 3
        cache.extend(slot, 1)
    assert cache.groups[0].pool.allocations == 15
    from tiny_inference_server_b200.cache.pages import CacheError
    cache.truncate(slot, 50)
    with pytest.raises(CacheError):
        cache.truncate(slot, 40)


# ------------------------------------------------------------------------------------------------
# the engine's plumbing on the CPU, the kernels replaced by plain references
# ------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", ["M1", "M2", "M4"])
@pytest.mark.parametrize("mode", ["whole", "tail", "chunks", "mixed"])
def test_replay_cpu(name, mode, tmp_path, tmp_path_factory, ref_ops):
    raw, page, folder, seqs, ref, _, _ = _setup(name, tmp_path_factory)
    seqs = {k: v for k, v in seqs.items() if len(v) <= 45}
    _replay_and_compare(raw, page, folder, seqs, ref, _steps(mode, seqs, max_live=3), str(tmp_path / "out"), "float32", "cpu",
                        TOL["float32"], max_live=3, poison=True)


def _check_layers(folder, page, toks, c, W, device):
    """The residual stream after every layer, read from the model's blocks one by one, against the plain layers."""
    from tiny_inference_server_b200.engine.batch import StepEntry
    _, layers = plain.plain_forward(c, W, toks, return_layers=True)
    runner = make_runner(folder, "float32", 256, page_size=page, max_live=1, cuda_graphs=False, device=device)
    seen = []
    for e in runner.model.entries:
        inner = e.block.forward

        def spy(stream, step, binding, *a, _inner=inner, **kw):
            _inner(stream, step, binding, *a, **kw)
            seen.append(stream.flush().clone())
        e.block.forward = spy
    slot = runner.add_request()
    runner.step([StepEntry(slot, list(toks), [len(toks) - 1])])
    runner.release(slot)
    assert len(seen) == layers.shape[0]
    for i, (got, want) in enumerate(zip(seen, layers)):
        err = float((got.double().cpu() - want).abs().max() / want.abs().max())
        assert err < 1e-4, f"stream after layer {i}: {err}"


def test_layers_of_the_stream_cpu(tmp_path_factory, ref_ops):
    raw, page, folder, seqs, _, c, W = _setup("M1", tmp_path_factory)
    _check_layers(folder, page, seqs["r3"], c, W, "cpu")


def plain_greedy(c, W, prompt, new):
    ids = list(prompt)
    for _ in range(new):
        ids.append(int(plain.plain_forward(c, W, ids)[-1].argmax()))
    return ids[len(prompt):]


def test_generate_cpu(tmp_path_factory, ref_ops):
    raw, page, folder, seqs, _, c, W = _setup("M2", tmp_path_factory)
    prompts = [seqs["r1"], seqs["r0"], seqs["r4"]]
    want = [plain_greedy(c, W, p, 6) for p in prompts]
    sp = SamplingParams(max_new_tokens=6, temperature=0.0, ignore_eos=True)
    eng = Engine.from_folder(folder, EngineConfig(dtype="float32", page_size=page, num_pages=20, max_batch=2, device="cpu",
                                                  max_tokens_per_step=7, cuda_graphs=False))
    assert eng.generate(prompts, sp) == want
    assert eng.runner.cache.drained()


# ------------------------------------------------------------------------------------------------
# every mechanism alone, with planted inputs
# ------------------------------------------------------------------------------------------------

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
MECH_TOL = {"float32": 2e-5, "bfloat16": 3e-2}


def _close(got, ref, tol, what):
    got = got.detach().double().cpu()
    err = float((got - ref).abs().max() / max(float(ref.abs().max()), 1e-9))
    assert err < tol, f"{what}: relative error {err}"


def _round(t, dtype):
    return t.to(DT[dtype]).to(torch.float64)


def _run_mixers(mixers, inputs, portions, page, dtype, device, pages=None):
    """Feeds ``inputs`` ({request: (L, width)}) to the mixers through a cache manager and the step layout of the engine;
    ``portions``: a list of steps, each a list of (request, rows).  The first mixer's plane is everybody's; every mixer has a
    state of its own if it asks for one.  The requests' slots are given back at the end.  Returns {request: [output of every
    mixer (L, columns)]} in float64."""
    from tiny_inference_server_b200.engine.batch import StepEntry, build_step
    dev = torch.device(device)
    longest = max(len(x) for x in inputs.values())
    n_pages = pages or sum((len(x) + page - 1) // page for x in inputs.values()) + 1
    states = {f"m{i}": mx.state_spec() for i, mx in enumerate(mixers) if mx.state_spec() is not None}
    cache = CacheManager([mixers[0].kv_spec()], states, page_size=page, num_pages=n_pages, max_slots=len(inputs) + 1,
                         max_positions=longest + page, dtype=DT[dtype], device=dev, debug_poison=True)
    import random
    for grp in cache.groups:
        grp.pool.shuffle(random.Random(1))
    for t in cache.states.values():
        t.fill_(7.0)                                        # what a slot held before must not show
    bindings = [LayerBinding(state=cache.states.get(f"m{i}")) for i in range(len(mixers))]
    if cache.groups:
        grp, ref = cache.groups[0], cache.plane_refs[0]
        for b in bindings:
            b.kv_plane, b.kv_group, b.k_pages, b.v_pages = grp.plane(ref.index), 0, grp.key_pages(ref.index), grp.value_pages(ref.index)
    planners = []
    for mx in mixers:
        planners += [p for p in mx.step_planners() if all(p.key != q.key for q in planners)]
    fault = torch.zeros(4, dtype=torch.int32, device=dev)
    slots = {rid: cache.admit() for rid in inputs}
    fed = {rid: 0 for rid in inputs}
    out = {rid: [None] * len(mixers) for rid in inputs}
    for step_entries in portions:
        entries = [StepEntry(slots[rid], [0] * n, []) for rid, n in step_entries]
        starts = [cache.extend(slots[rid], n) for rid, n in step_entries]
        assert starts == [fed[rid] for rid, _ in step_entries]
        cache.sync_tables()
        step, _, _ = build_step(entries, starts, [0], [g.table_dev for g in cache.groups], [page] * len(cache.groups), fault, dev, 1,
                                planners=planners)
        x = torch.cat([inputs[rid][fed[rid]:fed[rid] + n] for rid, n in step_entries]).to(DT[dtype]).to(dev)
        for i, mx in enumerate(mixers):
            y = mx.forward(x.clone(), step, bindings[i]).double().cpu()
            at = 0
            for rid, n in step_entries:
                if out[rid][i] is None:
                    out[rid][i] = torch.zeros(len(inputs[rid]), y.shape[1], dtype=torch.float64)
                out[rid][i][fed[rid]:fed[rid] + n] = y[at:at + n]
                at += n
        for rid, n in step_entries:
            fed[rid] += n
    assert int(fault[0]) == 0
    for rid in inputs:
        assert fed[rid] == len(inputs[rid])
        cache.release(slots[rid])
    cache.check()
    assert cache.drained()
    return out


def _steps_of_two(L, other):
    """Portions of request "a" (L rows) of changing size, some of them single rows, with portions of "b" (``other`` rows)
    beside some of them."""
    cuts, steps, fa, fb, i = (70, 2, 1, 16, 1, 100, 3, 1), [], 0, 0, 0
    while fa < L or fb < other:
        entries = []
        if fa < L:
            n = min(cuts[i % len(cuts)], max(1, L - 9 - fa)) if fa < L - 9 else 1
            entries.append(("a", n))
            fa += n
        if fb < other and i % 3 != 1:
            n = min((1, 9, 1, 33)[i % 4], other - fb)
            entries.insert(i % 2, ("b", n))
            fb += n
        if entries:
            steps.append(entries)
        i += 1
    return steps


# ---- attention: chunks, bounded scores, sinks, head gates, heads normed as a whole -----------------------------------

def _attention_mixers(m, readers, eps, dtype, device, width):
    """The mixer of ``m`` and those of ``readers`` on one plane, with projections that pick columns of the input (queries, keys,
    values, then the gates), norm weights and sinks of their own and the identity as output; (mixers, plain weights)."""
    from tiny_inference_server_b200.parts.normed_attention import NormedRotaryAttention
    from tiny_inference_server_b200.parts.positions import RotaryBanded
    g = torch.Generator().manual_seed(m["dim"])
    ctx = BuildContext(torch.device(device), DT[dtype])
    sizes = [(x.get("mask") or {}).get("size") for x in [m] + readers]
    keep = () if any(s is None for s in sizes) else tuple(sizes)
    out, weights = [], []
    for x, size in zip([m] + readers, sizes):
        rot, pos = x.get("rot"), None
        if rot:
            pos = RotaryBanded(x["dim"], rot["base"], 512, scaling=rot.get("scaling"), rotary_dim=rot["dims"])
            pos.load({}, ctx)
        mixer = NormedRotaryAttention(width, x["heads"], x["kv_heads"], x["dim"], x["vdim"], x["scale"], eps, pos, window=size,
                                      qk_norm="whole", reads_cache=x is not m, chunked=True, cache_chunks=keep,
                                      softcap=x.get("softcap"), head_gate=True, prefix="")
        nq, nk, nv, no = x["heads"] * x["dim"], x["kv_heads"] * x["dim"], x["kv_heads"] * x["vdim"], x["heads"] * x["vdim"]
        W, at = {}, 0
        for name, n in (("q", nq), ("k", nk), ("v", nv), ("g", x["heads"])):
            W[name] = torch.zeros(n, width, dtype=torch.float64)
            W[name][torch.arange(n), at + torch.arange(n)] = 1.0
            at += n
        W["q.norm"] = _round(1 + 0.2 * torch.randn(nq, generator=g), "bfloat16")
        W["k.norm"] = _round(1 + 0.2 * torch.randn(nk, generator=g), "bfloat16")
        W["o"] = torch.eye(no, dtype=torch.float64)
        W["sink"] = torch.randn(x["heads"], generator=g).double()
        W["sink"][0] = 2.5
        load = dict(W, o=torch.zeros(width, no, dtype=torch.float64))
        load["o"][:no] = W["o"]
        mixer.load({k: v.float() for k, v in load.items() if not (x is not m and k[0] in "kv")}, ctx)
        out.append(mixer)
        weights.append(W)
    return out, weights


def _planted(m, L, width, dtype, seed, size):
    """A random input in which some queries look like one key each: the first key of the query's chunk, the last one of the
    chunk before (not seen), the sequence's first token, the neighbour.  Query and key lie in the channel that turns most
    slowly (or not at all) and nowhere else.  Returns (input, [(query, key)])."""
    g = torch.Generator().manual_seed(seed)
    nq, nk, D = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["dim"]
    u = _round(torch.randn(L, width, generator=g), dtype)
    pairs, used = [], set()
    C = size or 10 ** 9
    edges = [(c, c - 1) for c in range(C, L, C)][:2] + [(min(c + C, L) - 1, c) for c in range(0, L, C)][:2] + [(L - 1, (L - 1) - (L - 1) % C)]
    for p, j in edges + [(L - 3, (L - 3) - (L - 3) % C), (2 * L // 3, 2 * L // 3 - 1), (L // 2, L // 2 - 17), (L // 3, 0), (5, 4)]:
        if 0 <= j < p and not {p, j} & used:
            pairs.append((p, j))
            used.update((p, j))
    for n, (p, j) in enumerate(pairs):
        c = D - 1 - n % max(1, D - (m.get("rot") or {"dims": 0})["dims"])
        u[p, :nq] = 0.0
        u[p, c:nq:D] = 1.5
        u[j, nq:nq + nk] = 0.0
        u[j, nq + c:nq + nk:D] = 1.5
    return u, pairs


ATTENTION_CASES = [          # heads, kv heads, dim, vdim, rotated, chunk, page, scaling, bound
    (4, 2, 32, 32, 16, 37, 16, None, 9.0),
    (8, 1, 64, 64, 64, 70, 16, (4.0, 1.0, 4.0, 64), 12.0),
    (2, 2, 128, 128, 128, 130, 32, None, 8.0),
    (6, 2, 48, 48, 24, 1, 8, None, 6.0),
    (6, 2, 48, 48, 24, 2, 8, (3.0, 1.0, 2.0, 50), None),
    (3, 3, 10, 6, 4, 19, 4, None, 7.0),
    (4, 1, 32, 48, None, 33, 16, None, 10.0),
    (20, 1, 16, 16, 8, 50, 16, None, 9.0),
    (12, 1, 80, 80, 8, 64, 16, None, None),
    (4, 4, 256, 256, 128, 90, 16, None, 6.0),
    (4, 2, 64, 64, 32, None, 16, (8.0, 1.0, 4.0, 128), 11.0),
    (6, 3, 24, 40, 10, None, 5, None, 5.0),
    (2, 1, 64, 64, 62, 128, 64, None, 12.0),
    (8, 2, 96, 96, 96, 100, 16, (4.0, 1.0, 4.0, 200), 6.5),
]


def _check_attention(case, dtype, device):
    H, G, dim, vdim, rot, size, page, scaling, cap = case
    _, m = _attn(H, G, dim, vdim, size, rot=rot, scaling=scaling, softcap=cap, scale=14.0 / dim)
    eps = 1e-4
    width = max(H * dim + G * (dim + vdim) + H, H * vdim)
    mixers, weights = _attention_mixers(m, [], eps, dtype, device, width)
    L, other = 300, 90
    u, pairs = _planted(m, L, width, dtype, H * 10 + dim, size)
    b, _ = _planted(m, other, width, dtype, H * 10 + dim + 1, size)
    want = {rid: plain.attention(x, weights[0], "", m, eps)[0] for rid, x in (("a", u), ("b", b))}
    got = _run_mixers(mixers, {"a": u, "b": b}, _steps_of_two(L, other), page, dtype, device)
    tol = MECH_TOL[dtype]
    no = H * vdim
    _close(got["a"][0][:, :no], want["a"], tol, "attention in portions")
    _close(got["b"][0][:, :no], want["b"], tol, "the request beside it")
    for p, j in pairs:
        _close(got["a"][0][p, :no], want["a"][p], 2 * tol, f"the query at {p}, which looks for the key at {j}")
    # what is tested matters: other chunks, other bounds, no sink, no gate, a norm per head are far outside the tolerance
    rows = want["a"].abs().max(-1).values

    def off(changed, w=weights[0]):
        return float(((plain.attention(u, w, "", changed, eps)[0] - want["a"]).abs().max(-1).values / rows).max())
    if size:
        assert off(dict(m, mask={"size": size + 1})) > 5 * tol
        if size > 1:
            assert off(dict(m, mask={"size": size - 1})) > 5 * tol
    if cap:
        assert off(dict(m, softcap=None)) > 5 * tol or size == 1 or size == 2
    assert off(m, dict(weights[0], sink=torch.full((H,), -1e9, dtype=torch.float64))) > 5 * tol
    assert off(m, dict(weights[0], g=weights[0]["g"] * 0)) > 5 * tol


@pytest.mark.parametrize("case", [c for c in ATTENTION_CASES if c[2] <= 48])
def test_attention_chunks_bounds_and_planted_keys_cpu(case, ref_ops):
    _check_attention(case, "float32", "cpu")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ATTENTION_CASES)
def test_attention_chunks_bounds_and_planted_keys(case, dtype):
    from tiny_inference_server_b200.kernels import ops
    before = dict(ops.calls)
    _check_attention(case, dtype, "cuda:0")
    if dtype == "bfloat16" and case[2] == case[3] and case[2] % 16 == 0 and case[0] // case[1] <= 16:
        assert ops.calls["attn_keys"] > before.get("attn_keys", 0)
        if case[2] in (64, 128):
            assert ops.calls["attn_tc"] > before.get("attn_tc", 0)


def _check_readers(dims, dtype, device):
    """Layers that read another layer's keys with chunks larger and smaller than its own: a plane that gave pages back by its
    owner's chunk would show poison to the other reader."""
    H, G, dim, vdim, page = dims
    _, owner = _attn(H, G, dim, vdim, 11, rot=dim // 2 * 2, scale=14.0 / dim)
    readers = [dict(owner, mask={"size": 60}, kv_from=0, scale=10.0 / dim, softcap=6.0), dict(owner, mask={"size": 4}, kv_from=0)]
    eps, L = 1e-4, 200
    width = max(H * dim + G * (dim + vdim) + H, H * vdim)
    mixers, weights = _attention_mixers(owner, readers, eps, dtype, device, width)
    u, _ = _planted(owner, L, width, dtype, 3, 60)
    want, held = plain.attention(u, weights[0], "", owner, eps)
    no = H * vdim
    wants = [want] + [plain.attention(u, w, "", m, eps, held)[0] for m, w in zip(readers, weights[1:])]
    short = _round(torch.randn(13, width, generator=torch.Generator().manual_seed(8)), dtype)
    # few pages: what lies before the earliest chunk is given back and used again
    pages = (60 + 40) // page + 6
    steps = [[("a", n)] for n in (40, 1, 2, 33, 1, 1, 17, 5)] + [[("b", 6), ("a", 1)], [("b", 1), ("a", 2)]] + \
        [[("a", 1)]] * 97 + [[("b", 6)]]
    got = _run_mixers(mixers, {"a": u, "b": short}, steps, page, dtype, device, pages=pages)
    for i, w in enumerate(wants):
        _close(got["a"][i][:, :no], w, MECH_TOL[dtype], f"layer {i} over the shared plane")
    assert float((plain.attention(u, weights[1], "", dict(readers[0], mask={"size": 11}), eps, held)[0] - wants[1]).abs().max()) \
        > 5 * MECH_TOL[dtype] * float(wants[1].abs().max())


def test_readers_with_chunks_of_their_own_cpu(ref_ops):
    _check_readers((4, 2, 16, 16, 4), "float32", "cpu")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dims", [(4, 2, 16, 16, 4), (8, 2, 64, 64, 16), (4, 1, 32, 48, 8), (3, 3, 12, 7, 4)])
def test_readers_with_chunks_of_their_own(dims, dtype):
    _check_readers(dims, dtype, "cuda:0")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("permuted", [False, True])
@pytest.mark.parametrize("H,G,dim,vdim,rot,interleaved,page", [
    (4, 2, 32, 32, 32, True, 16), (3, 1, 96, 64, 40, True, 4), (2, 2, 16, 16, 6, False, 8), (5, 0, 48, 48, 48, True, 16),
    (6, 3, 128, 128, 0, True, 16), (32, 8, 128, 128, 128, True, 16), (40, 2, 512, 64, 256, True, 16), (3, 3, 10, 6, 10, True, 5)])
def test_norm_of_all_heads_then_rotation(dtype, permuted, H, G, dim, vdim, rot, interleaved, page):
    import kernel_refs
    from tiny_inference_server_b200.kernels import ops
    if permuted and (dim % 8 or vdim % 8):
        pytest.skip("rows of whole 16-byte chunks only")
    g = torch.Generator().manual_seed(H + dim)
    n, n_pages = 14, 12
    cols = H * dim + G * (dim + vdim)
    ld = (cols + 7) // 8 * 8
    x = torch.randn(n, ld, generator=g).to(DT[dtype])
    positions = torch.tensor(list(range(3, 10)) + list(range(7)), dtype=torch.int32)
    row_slot = torch.tensor([1] * 7 + [0] * 5 + [-1] * 2, dtype=torch.int32)
    per = 16 // page + 1
    table = torch.randperm(n_pages, generator=g)[:2 * per].to(torch.int32).view(2, per)
    cos, sin = torch.randn(40, rot // 2, generator=g), torch.randn(40, rot // 2, generator=g)
    norm_ = torch.sqrt(cos * cos + sin * sin)
    cos, sin = (cos / norm_, sin / norm_) if rot else (None, None)
    w = 1 + 0.3 * torch.randn((H + G) * dim, generator=g)
    k = torch.zeros(n_pages, max(G, 1), page, dim, dtype=DT[dtype])
    v = torch.zeros(n_pages, max(G, 1), page, vdim, dtype=DT[dtype])
    xr, kr, vr = x.clone(), k.clone(), v.clone()
    kernel_refs.rotate_norm_store(xr, H, G, dim, vdim, cos, sin, interleaved, True, 1e-4, kr, vr, table, positions, row_slot, page,
                                  None, permuted=permuted, whole_weight=w)
    xd, kd, vd, fd = x.cuda(), k.cuda(), v.cuda(), torch.zeros(4, dtype=torch.int32, device="cuda")
    ops.rotate_norm_store(xd, H, G, dim, vdim, cos.cuda() if rot else None, sin.cuda() if rot else None, interleaved, True, 1e-4,
                          kd if G else None, vd if G else None, table.cuda(), positions.cuda(), row_slot.cuda(), page, fd,
                          permuted=permuted, whole_weight=w.cuda())
    tol = {"float32": 1e-5, "bfloat16": 1e-2}[dtype]
    _close(xd[:, :H * dim], xr[:, :H * dim].double(), tol, "queries")
    assert torch.equal(xd[:, H * dim:cols].cpu(), x[:, H * dim:cols]), "keys and values of the rows were written"
    if G:
        _close(kd, kr.double(), tol, "key rows")
        assert torch.equal(vd.cpu(), vr), "value rows"
    assert int(fd[0]) == 0


# ---- the selective scan ------------------------------------------------------------------------------------------------

SCAN_CASES = [(24, 40, 8, 5, 4), (64, 128, 16, 4, 4), (40, 27, 5, 3, 2), (32, 64, 1, 8, 1), (48, 96, 32, 7, 3), (24, 33, 50, 2, 16),
              (16, 20, 100, 2, 2), (16, 12, 200, 1, 4), (64, 300, 3, 20, 4), (96, 512, 64, 6, 4)]      # width, inner, state, rank, taps


def _scan_setup(case, dtype, device):
    from tiny_inference_server_b200.parts.selective_scan import SelectiveScan
    width, inner, state, rank, taps = case
    g = torch.Generator().manual_seed(inner + state)
    part = SelectiveScan(width, inner, state, rank, taps)
    W = {}
    for p in part.walk():
        for name, spec in p.expected_tensors().items():
            rnd, uni = torch.randn(*spec.shape, generator=g), torch.rand(*spec.shape, generator=g)
            t = {"A_log": uni * 7 - 6, "dt.b": uni * 3 - 2.5, "D": rnd, "conv": rnd / math.sqrt(taps), "conv.b": rnd * 0.3}.get(
                name, rnd / math.sqrt(spec.shape[-1]))
            W[name] = _round(t, "bfloat16")
    ctx = BuildContext(torch.device(device), DT[dtype])
    for p in part.walk():
        p.load({k: v.float() for k, v in W.items()}, ctx)
    return part, W, {"inner": inner, "state": state, "dt_rank": rank, "conv": taps}


def _check_scan(case, dtype, device):
    part, W, m = _scan_setup(case, dtype, device)
    g = torch.Generator().manual_seed(4)
    L, other = 230, 41
    x = {rid: _round(torch.randn(n, case[0], generator=g), dtype) for rid, n in (("a", L), ("b", other))}
    x["a"][3] *= 12.0                                       # an event that the slow states still hold at the end
    want = {rid: plain.selective_scan_mixer(v, W, "", m, 0.0) for rid, v in x.items()}
    tol = {"float32": 5e-5, "bfloat16": 4e-2}[dtype]
    got = _run_mixers([part], x, _steps_of_two(L, other), 16, dtype, device)
    _close(got["a"][0], want["a"], tol, "scan in portions")
    _close(got["b"][0], want["b"], tol, "the request beside it")
    alone = _run_mixers([part], {"a": x["a"]}, [[("a", L - 40)]] + [[("a", 1)]] * 40, 16, dtype, device)
    _close(alone["a"][0], want["a"], tol, "a prompt, then one by one")
    quiet = x["a"].clone()
    quiet[3] /= 12.0
    late = want["a"][-20:]
    rounding = float((alone["a"][0][-20:] - late).abs().max())
    assert float((plain.selective_scan_mixer(quiet, W, "", m, 0.0)[-20:] - late).abs().max()) > 2 * rounding or m["state"] < 3


@pytest.mark.parametrize("case", SCAN_CASES[:5])
def test_selective_scan_cpu(case, ref_ops):
    _check_scan(case, "float32", "cpu")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", SCAN_CASES)
def test_selective_scan(case, dtype):
    _check_scan(case, dtype, "cuda:0")


@gpu
@pytest.mark.parametrize("fine", [0, 1 << 30])
@pytest.mark.parametrize("channels,states", [(5, 1), (40, 3), (64, 4), (100, 16), (130, 17), (33, 32), (20, 33), (70, 64), (9, 128), (17, 256)])
def test_selective_scan_kernel_alone(channels, states, fine, monkeypatch):
    """The kernel in 32-bit, every number of lanes and states a lane, portions of one to seventy rows over three slots, states
    kept in a wider row than they need."""
    import kernel_refs
    from tiny_inference_server_b200.kernels import ops
    monkeypatch.setattr(ops, "SCAN_FINE_MAX_CHANNELS", fine)
    g = torch.Generator().manual_seed(channels)
    slots, n = 3, 104
    row_slot = torch.tensor([1] * 33 + [0] + [2] * 70, dtype=torch.int32)
    row_last = torch.tensor([32] * 33 + [33] + [103] * 70, dtype=torch.int32)
    first = torch.tensor([0, 33, 34], dtype=torch.int32)

    def rand(*s):
        return torch.randn(*s, generator=g)
    x, z, dt, bc = rand(n, channels + 3), rand(n, channels), rand(n, channels) - 1.0, rand(n, 2 * states + 1)
    bias, a_log, skip = rand(channels), torch.rand(channels, states, generator=g) * 5 - 4, rand(channels)
    state = rand(slots, channels * states + 7)
    args = lambda t: (t(x)[:, :channels], t(dt), t(bias), t(a_log), t(bc)[:, :states], t(bc)[:, states:2 * states], t(skip), t(z))  # noqa: E731
    sr, outr = state.clone(), torch.zeros(n, channels)
    kernel_refs.selective_scan(*args(lambda t: t), sr, outr, row_slot, row_last)
    for segments in (None, (first.cuda(), 3)):
        sd, outd = state.cuda(), torch.zeros(n, channels, device="cuda")
        ops.selective_scan(*args(lambda t: t.cuda()), sd, outd, row_slot.cuda(), row_last.cuda(), segments=segments)
        _close(outd, outr.double(), 2e-5, "outputs")
        _close(sd, sr.double(), 2e-5, "states")
        assert torch.equal(sd[:, channels * states:].cpu(), state[:, channels * states:]), "beyond the states"


# ---- the time mixer ----------------------------------------------------------------------------------------------------

MIX_CASES = [(24, 2, 16, 5), (64, 3, 32, 8), (40, 3, 10, 3), (48, 2, 64, 16), (32, 1, 128, 8), (40, 2, 96, 6), (56, 2, 48, 8),
             (128, 4, 64, 64), (16, 1, 200, 4)]      # width, heads, dim, rank


def _mix_setup(case, dtype, device):
    from tiny_inference_server_b200.parts.time_mix import TimeMix
    width, heads, dim, rank = case
    g = torch.Generator().manual_seed(width + dim)
    eps = 1e-4
    part = TimeMix(width, heads, dim, rank, eps)
    W = {}
    for name, spec in part.expected_tensors().items():
        rnd, uni = torch.randn(*spec.shape, generator=g), torch.rand(*spec.shape, generator=g)
        t = uni * 1.4 - 0.2 if name.startswith("mu.") else \
            {"w0": uni * 9 - 8, "u": rnd, "norm": 1 + 0.2 * rnd}.get(name, rnd / math.sqrt(spec.shape[-1]))
        W[name] = _round(t, "bfloat16")
    part.load({k: v.float() for k, v in W.items()}, BuildContext(torch.device(device), DT[dtype]))
    return part, W, {"heads": heads, "dim": dim}, eps


def _check_mix(case, dtype, device):
    part, W, m, eps = _mix_setup(case, dtype, device)
    g = torch.Generator().manual_seed(4)
    L, other = 230, 41
    x = {rid: _round(torch.randn(n, case[0], generator=g), dtype) for rid, n in (("a", L), ("b", other))}
    x["a"][3] *= 12.0                                       # a token that slow channels still hold at the end
    want = {rid: plain.time_mix(v, W, "", m, eps) for rid, v in x.items()}
    tol = {"float32": 5e-5, "bfloat16": 4e-2}[dtype]
    got = _run_mixers([part], x, _steps_of_two(L, other), 16, dtype, device)
    _close(got["a"][0], want["a"], tol, "time mixer in portions")
    _close(got["b"][0], want["b"], tol, "the request beside it")
    alone = _run_mixers([part], {"a": x["a"]}, [[("a", L - 40)]] + [[("a", 1)]] * 40, 16, dtype, device)
    _close(alone["a"][0], want["a"], tol, "a prompt, then one by one")
    # what the mechanism consists of matters: the bonus, the token before, the far token
    scale = float(want["a"].abs().max())
    assert float((plain.time_mix(x["a"], dict(W, u=W["u"] * 0), "", m, eps) - want["a"]).abs().max()) > 2 * tol * scale
    assert float((plain.time_mix(x["a"], dict(W, **{"mu.v": W["mu.v"] * 0}), "", m, eps) - want["a"]).abs().max()) > 2 * tol * scale
    quiet = x["a"].clone()
    quiet[3] /= 12.0
    rounding = float((alone["a"][0][-20:] - want["a"][-20:]).abs().max())
    assert float((plain.time_mix(quiet, W, "", m, eps)[-20:] - want["a"][-20:]).abs().max()) > 2 * rounding


@pytest.mark.parametrize("case", MIX_CASES[:4])
def test_time_mixer_cpu(case, ref_ops):
    _check_mix(case, "float32", "cpu")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", MIX_CASES)
def test_time_mixer(case, dtype):
    from tiny_inference_server_b200.kernels import ops
    before = ops.calls["gemm_skinny_groups"]
    _check_mix(case, dtype, "cuda:0")
    if dtype == "bfloat16" and case[0] % 8 == 0 and case[1] * case[2] % 64 == 0:
        assert ops.calls["gemm_skinny_groups"] > before            # decode rows: all products in one launch


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d", [8, 13, 64, 1000, 1536])
def test_token_shift_kernel(d, dtype):
    import kernel_refs
    from tiny_inference_server_b200.kernels import ops
    g = torch.Generator().manual_seed(d)
    row_slot = torch.tensor([1] * 5 + [0] + [-1] + [2] * 2, dtype=torch.int32)
    row_last = torch.tensor([4] * 5 + [5] + [6] + [8] * 2, dtype=torch.int32)
    x, mu = torch.randn(9, d, generator=g).to(DT[dtype]), torch.rand(5, d, generator=g)
    state = torch.randn(3, d + 5, generator=g)
    sr = state.clone()
    want = kernel_refs.token_shift(x, mu, sr, row_slot, row_last)
    sd = state.cuda()
    got = ops.token_shift(x.cuda(), mu.cuda(), sd, row_slot.cuda(), row_last.cuda())
    live = row_slot >= 0
    _close(got.cpu()[live], want[live].double(), {"float32": 1e-6, "bfloat16": 1e-2}[dtype], "mixes")
    assert torch.equal(sd.cpu(), sr), "the last inputs"


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,K,N,M", [(1, 64, 64, 8), (8, 1536, 1536, 64), (3, 200, 128, 16), (17, 512, 192, 24), (32, 96, 64, 0), (40, 64, 128, 8),
                                     (5, 40, 30, 5), (300, 128, 64, 16)])
def test_products_side_by_side(n, K, N, M, dtype):
    from tiny_inference_server_b200.kernels import ops
    if M == 0:
        M = 8
    g = torch.Generator().manual_seed(n + K)
    a = _round(torch.randn(n, 5, K, generator=g), dtype)
    w = _round(torch.randn(4, K, N, generator=g) / math.sqrt(K), dtype)
    wl = _round(torch.randn(K, M, generator=g) / math.sqrt(K), dtype)
    for act in ("tanh", None):
        out, last = ops.gemm_side_by_side(*(t.to(DT[dtype]).cuda() for t in (a, w, wl)), act=act)
        tol = {"float32": 1e-5, "bfloat16": 1e-2}[dtype]
        _close(out, torch.einsum("ngk,gkj->ngj", a[:, :4], w).reshape(n, -1), tol, "side by side")
        want = a[:, 4] @ wl
        _close(last, torch.tanh(want) if act else want, tol, "the last one")


# ---- norms behind the sublayers, the mixture ---------------------------------------------------------------------------

@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d", [(3, 64), (37, 40), (1, 1000), (1030, 192), (2048, 1536), (2, 13)])
def test_norm_behind_a_sublayer_and_the_stream_as_it_is(dtype, n, d):
    from tiny_inference_server_b200.parts.norms import RMSNormMeanEps, StreamAsIs
    from tiny_inference_server_b200.parts.stream import ResidualStream
    g = torch.Generator().manual_seed(n + d)
    ctx = BuildContext(torch.device("cuda:0"), DT[dtype])
    w = _round(1 + 0.2 * torch.randn(d, generator=g), "bfloat16")
    post, as_is = RMSNormMeanEps(d, 1e-4, prefix="n", weight_name="", gain=0.37), StreamAsIs(d)
    post.load({"n": w.float()}, ctx)
    as_is.load({}, ctx)
    x = torch.randn(n, d, generator=g) * 3
    delta = torch.randn(n, d, generator=g).to(DT[dtype]) * 5
    stream = ResidualStream(x.cuda())
    _close(stream.normed(as_is), x.to(DT[dtype]).double(), 1e-6, "the stream as it is")
    stream.add(delta.cuda(), post=post)
    want = x.double() + 0.37 * plain.rms_norm(delta.double(), w, 1e-4)
    h = stream.normed(as_is)
    assert h.dtype == DT[dtype]
    _close(stream.values, want, 1e-6, "the stream with its update")
    _close(h, want, {"float32": 1e-6, "bfloat16": 5e-3}[dtype], "what the next sublayer reads")
    stream.add(delta.cuda(), post=post)
    _close(stream.flush(), want + 0.37 * plain.rms_norm(delta.double(), w, 1e-4), 1e-6, "the stream at the end of a layer")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d,F,E,top", [(3, 48, 40, 6, 2), (1, 64, 96, 16, 4), (40, 64, 32, 12, 3), (300, 128, 64, 8, 4), (700, 192, 96, 16, 4),
                                         (600, 128, 128, 8, 2), (50, 40, 24, 5, 5), (2000, 64, 64, 4, 1), (9, 32, 32, 1, 1)])
def test_experts_whose_inputs_are_weighed(dtype, n, d, F, E, top):
    """The whole mixture against the plain one: few rows (a dot product per element), a hundred pairs (tiles on the tensor
    cores), a thousand (tcgen05 tiles)."""
    from tiny_inference_server_b200.kernels import ops
    from tiny_inference_server_b200.parts.feed_forward import RoutedExperts
    g = torch.Generator().manual_seed(n + d)
    f = _moe(F, E, top)
    part = RoutedExperts(d, F, E, top, scores="sigmoid", correction=False, renorm=False, weigh_input=True)
    W = {name: _round(torch.randn(*spec.shape, generator=g) * 1.5 / math.sqrt(spec.shape[1]), dtype)
         for name, spec in part.expected_tensors().items()}
    x = _round(torch.randn(n, d, generator=g), dtype)
    want = plain.expert_mixture(x, W, "", f)
    part.load({k: v.float() for k, v in W.items()}, BuildContext(torch.device("cuda:0"), DT[dtype]))
    chosen, weights = plain.route(x, W["router"], f["router"])
    noisy, _ = plain.route(x * (1 + 1e-4), W["router"] + 1e-4 * torch.randn(W["router"].shape, generator=g).double(), f["router"])
    clear = (chosen.sort(-1).values == noisy.sort(-1).values).all(-1)         # rows whose choice hangs on a rounding are left out
    assert int(clear.sum()) >= max(1, int(0.9 * n))
    got_chosen, got_weights, _ = ops.moe_route(x.to(DT[dtype]).cuda(), part.w_router, None, None, 0, 0, top, renorm=False)
    assert torch.equal(got_chosen.cpu().long()[clear].sort(-1).values, chosen[clear].sort(-1).values)
    _close(got_weights.cpu()[clear].sort(-1).values, weights[clear].sort(-1).values, 1e-5, "weights")
    before = dict(ops.calls)
    out = part.forward(x.to(DT[dtype]).cuda())
    tol = {"float32": 2e-5, "bfloat16": 3e-2}[dtype]
    _close(out[clear.cuda()], want[clear], tol, "mixture")
    # the weight outside the unit is another function
    outside = torch.zeros_like(want)
    for e in range(E):
        for j in range(top):
            rows = (chosen[:, j] == e).nonzero().flatten()
            if len(rows):
                outside[rows] += weights[rows, j:j + 1] * plain.silu_unit(x[rows], W, f"e{e}.")
    assert float((outside - want).abs().max()) > 3 * tol * float(want.abs().max())
    if dtype == "bfloat16" and n * top >= 1024 and d % 64 == 0 and F % 64 == 0:
        assert ops.calls["moe_grouped_tc"] == before.get("moe_grouped_tc", 0) + 1
    elif dtype == "bfloat16" and n * top >= 96 and d % 32 == 0 and F % 32 == 0:
        assert ops.calls["moe_grouped"] == before.get("moe_grouped", 0) + 1


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,K,F", [(1, 64, 96), (8, 192, 320), (20, 128, 64), (30, 2048, 512), (3100, 64, 128), (5, 40, 50)])
def test_clamped_unit_without_biases(dtype, n, K, F):
    from tiny_inference_server_b200.kernels import ops
    from tiny_inference_server_b200.parts.feed_forward import SwiGLU
    g = torch.Generator().manual_seed(n + F)
    x = _round(torch.randn(n, K, generator=g), dtype)
    W = {k: _round(torch.randn(*((K, F) if k == "down" else (F, K)), generator=g) * 2 / math.sqrt(F if k == "down" else K), dtype)
         for k in ("gate", "up", "down")}
    want = plain.clamped_unit(x, W, "", 0.7)
    assert float((want - plain.clamped_unit(x, W, "", 1.0)).abs().max()) > 0.1
    part = SwiGLU(K, F, names={"gate": "gate", "up": "up", "down": "down"}, stored_out_in=True, form=ops.gate_clamped(0.7))
    part.load({k: v.float() for k, v in W.items()}, BuildContext(torch.device("cuda:0"), DT[dtype]))
    _close(part.forward(x.to(DT[dtype]).cuda()), want, {"float32": 2e-5, "bfloat16": 2e-2}[dtype], "clamped unit")


# ------------------------------------------------------------------------------------------------
# whole models on the device
# ------------------------------------------------------------------------------------------------

@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M1", "M2", "M3", "M4"])
@pytest.mark.parametrize("mode", ["whole", "tail", "chunks", "mixed"])
def test_replay_gpu(name, mode, dtype, tmp_path, tmp_path_factory):
    raw, page, folder, seqs, ref, _, _ = _setup(name, tmp_path_factory, dtype)
    steps = _steps(mode, seqs, max_live=3)
    runner = _replay_and_compare(raw, page, folder, seqs, ref, steps, str(tmp_path / "out"), dtype, "cuda:0", TOL[dtype], max_live=3,
                                 poison=(mode == "mixed"), shuffle=(mode == "mixed"), outliers=OUTLIERS[dtype], cap=OUTLIER_CAP[dtype])
    if mode == "mixed" and name == "M1":          # its requests are long enough for the pool to turn over
        pool = runner.cache.groups[0].pool
        assert pool.allocations > pool.num_pages, "the trace does not use pages again"


@gpu
@pytest.mark.parametrize("name", ["M1", "M3", "M4"])
def test_layers_of_the_stream_gpu(name, tmp_path_factory):
    raw, page, folder, seqs, _, c, W = _setup(name, tmp_path_factory)
    _check_layers(folder, page, seqs["r5"], c, W, "cuda:0")


def random_configuration(seed):
    """A configuration drawn at random: kinds, sizes, chunks, rotations, readers, feed-forwards, constants."""
    import random
    rng = random.Random(seed)
    pick = rng.choice
    width = pick([24, 32, 48, 64, 96, 128, 192])
    layers, owners = [], []
    for i in range(rng.randint(3, 6)):
        kind = pick(["attention", "attention", "mamba1", "wkv"])
        if kind == "mamba1":
            mixer = _scan(pick([24, 40, 64, 100, 192, 256]), pick([1, 4, 8, 16, 24, 64]), pick([1, 3, 8, 12, 16]), pick([1, 2, 3, 4, 6]))
        elif kind == "wkv":
            mixer = _mix(pick([1, 2, 3, 4]), pick([8, 16, 20, 32, 64, 96]))
        else:
            size = pick([None, 1, 3, 16, 17, 40, 64, 100, 250])
            cap = pick([None, 4.0, 15.0, 50.0])
            if owners and rng.random() < 0.4:
                j = pick(owners)
                m = dict(json.loads(json.dumps(layers[j][0][1])), kv_from=j, scale=pick([0.1, 0.2, 0.4]))
                m.pop("mask", None)
                m.pop("softcap", None)
                if size:
                    m["mask"] = {"size": size}
                if cap:
                    m["softcap"] = cap
                mixer = "attention", m
            else:
                kv, dim = pick([1, 2, 3]), pick([8, 16, 24, 32, 64, 80, 128])
                rot = pick([r for r in (2, 4, 8, 16, 24, 32, 64) if r <= dim] + [dim, None])
                mixer = _attn(kv * pick([1, 2, 3, 5]), kv, dim, pick([dim, dim, 16, 40]), size, rot=rot, softcap=cap,
                              scaling=pick([None, (4.0, 1.0, 4.0, 128), (2.0, 0.5, 8.0, 60)]), base=pick([100.0, 10000.0, 1e6]))
                owners.append(i)
        r = rng.random()
        if r < 0.1:
            mlp = None
        elif r < 0.45:
            mlp = _dense(pick([24, 32, 64, 100, 256]), pick([0.5, 1.0, 3.0]))
        else:
            mlp = _moe(pick([16, 32, 64, 96]), *pick([(4, 1), (4, 2), (8, 2), (16, 4), (6, 3), (3, 3), (1, 1)]))
        layers.append((mixer, mlp))
    return _cfg(rng.randint(40, 300), width, layers, eps=pick([1e-5, 1e-6, 1e-3]), mult=pick([0.4, 0.9, 1.0, 1.5]),
                cap=pick([None, 5.0, 20.0])), pick([4, 8, 16, 16, 32]), pick([1, 4, 7, 8, 24])


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10])
def test_configurations_drawn_at_random(seed, dtype, tmp_path):
    """Whatever config.json says runs without a change of code: configurations drawn at random, a mixed batch of five
    requests (one of them long) through three slots over shuffled pages."""
    raw, page, rank = random_configuration(seed)
    if dtype == "bfloat16":
        raw = all_chosen(raw)
    folder = make_folder(raw, 100 + seed, str(tmp_path / "m"), rank)
    c, W = plain.read_config(folder), plain.read_weights(folder)
    g = torch.Generator().manual_seed(seed)
    seqs = {f"r{i}": torch.randint(0, raw["vocab"], (n,), generator=g).tolist() for i, n in enumerate([1, 2, 45, 400, 130])}
    ref = {rid: plain.plain_forward(c, W, toks).numpy() for rid, toks in seqs.items()}
    steps = trace_tools.trace_mixed(seqs, max_live=3, prefill_sizes=(64, 2, 130, 17))
    _replay_and_compare(raw, page, folder, seqs, ref, steps, str(tmp_path / "out"), dtype, "cuda:0", TOL[dtype], max_live=3,
                        poison=True, shuffle=True, outliers=OUTLIERS[dtype], cap=OUTLIER_CAP[dtype])


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_two_slots_used_again_and_again(dtype, tmp_path, tmp_path_factory):
    """Eight requests through two slots over poisoned pages: a page that a request reads but does not hold shows."""
    raw, page, folder, seqs, ref, _, _ = _setup("M1", tmp_path_factory, dtype)
    steps = trace_tools.trace_mixed(seqs, max_live=2, prefill_sizes=(2, 7, 3, 2), skip_every=4)
    _replay_and_compare(raw, page, folder, seqs, ref, steps, str(tmp_path / "out"), dtype, "cuda:0", TOL[dtype], max_live=2,
                        poison=True, outliers=OUTLIERS[dtype], cap=OUTLIER_CAP[dtype])


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M3", "M4"])
def test_long_decoding(name, dtype, tmp_path, tmp_path_factory):
    """A short prompt, then 300 tokens one by one, replayed from a graph: every chunk passes over decoded tokens only."""
    raw, page, folder, _, _, c, W = _setup(name, tmp_path_factory, dtype)
    g = torch.Generator().manual_seed(9)
    toks = torch.randint(0, raw["vocab"], (305,), generator=g).tolist()
    ref = plain.plain_forward(c, W, toks).numpy()
    steps = trace_tools.trace_tail({"a": toks}, tail=300)
    runner = make_runner(folder, dtype, 320, page_size=page, max_live=1, debug_poison=True)
    out_dir = str(tmp_path / "out")
    TraceReplayer(runner, out_dir).run(json.dumps(s) for s in steps)
    assert runner.cache.drained()
    assert runner.graphs is not None and runner.graphs.replays > 250
    got = trace_tools.gather(steps, out_dir, raw["vocab"])
    errs = [rel_err(got["a"][p], ref[p]) for p in range(len(toks))]
    assert sum(e >= TOL[dtype] for e in errs) <= OUTLIERS[dtype] * len(errs), [(p, e) for p, e in enumerate(errs) if e >= TOL[dtype]]


@gpu
def test_generate_through_the_scheduler(tmp_path_factory):
    raw, page, folder, seqs, _, c, W = _setup("M3", tmp_path_factory)
    prompts = [seqs["r0"], seqs["r4"], seqs["r1"], seqs["r5"]]
    want = [plain_greedy(c, W, p, 10) for p in prompts]
    sp = SamplingParams(max_new_tokens=10, temperature=0.0, ignore_eos=True)
    for kw in (dict(max_batch=4, max_tokens_per_step=2048), dict(max_batch=2, max_tokens_per_step=9)):
        eng = Engine.from_folder(folder, EngineConfig(dtype="float32", page_size=page, num_pages=40, **kw))
        assert eng.generate(prompts, sp) == want
        assert eng.runner.cache.drained()
    eng = Engine.from_folder(folder, EngineConfig(dtype="bfloat16", page_size=page, num_pages=40, max_batch=4))
    out = eng.generate(prompts, sp)
    assert [len(o) for o in out] == [10] * 4 and eng.runner.cache.drained()


@gpu
def test_command_line_generation_with_chunking_and_preemption(tmp_path_factory):
    """Greedy tokens through ``python -m tiny_inference_server_b200.cli`` equal the plain implementation's: whole prompts; a
    token budget of five (portions beside decoding requests); and so few pages that requests are preempted and fed again."""
    from test_cli import _cli, _ids
    raw, page, folder, seqs, _, c, W = _setup("M1", tmp_path_factory)
    new = 8
    prompts = [seqs["r0"], seqs["r6"], seqs["r1"]]
    want = [plain_greedy(c, W, p, new) for p in prompts]
    args = ["--model", folder, "--greedy", "--ignore-eos", "--dtype", "float32", "--max-new-tokens", new,
            "--tokens-per-block", page, "--json"]
    for p in prompts:
        args += ["--prompt-ids", _ids(p)]
    r = _cli(*args)
    assert r.returncode == 0, r.stderr
    assert json.loads(r.stdout.strip().splitlines()[-1])["outputs"] == want
    r = _cli(*args, "--max-tokens-per-step", 5, "--max-batch", 2)
    assert r.returncode == 0, r.stderr
    assert json.loads(r.stdout.strip().splitlines()[-1])["outputs"] == want
    g = torch.Generator().manual_seed(31)
    prompts = [torch.randint(0, raw["vocab"], (page - 1,), generator=g).tolist() for _ in range(4)]
    want = [plain_greedy(c, W, p, new) for p in prompts]
    args = ["--model", folder, "--greedy", "--ignore-eos", "--dtype", "float32", "--max-new-tokens", new,
            "--tokens-per-block", page, "--json", "--num-pages", 5, "--plan", "cur", "--max-batch", 4,
            "--max-tokens-per-step", 16]
    for p in prompts:
        args += ["--prompt-ids", _ids(p)]
    r = _cli(*args)
    assert r.returncode == 0, r.stderr
    out = json.loads(r.stdout.strip().splitlines()[-1])
    assert out["outputs"] == want
    assert out["stats"]["preempts"] > 0 and out["stats"]["replays"] > 0
