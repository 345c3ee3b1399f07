"""The Lomutar architecture through the engine against the plain implementation (``plain_lomutar``): configuration and
weights, every mechanism alone with planted inputs, replays cut in every way, configurations drawn at random, slots and pages
used again, long decoding, generation through the scheduler and the command line."""
from __future__ import annotations

import json
import math
import os

import numpy as np
import pytest
import torch

import plain_lomutar as plain
import trace_tools
from tiny_inference_server_b200 import ConfigError, build_model, config_from_dict, config_from_folder
from tiny_inference_server_b200.api import Engine, SamplingParams
from tiny_inference_server_b200.config import EngineConfig, LomutarConfig
from tiny_inference_server_b200.trace import TraceReplayer, make_runner
from tiny_inference_server_b200.weights.loader import WeightError

gpu = pytest.mark.gpu


def _attn(heads, kv, dim, vdim, rot, size, factor=None, base=10000.0, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
         "scale": scale if scale is not None else 1.5 * dim ** -0.5}
    if factor:
        m["rot"]["scaling"] = {"factor": factor}
    if size:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, limit, experts, top, groups=None, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if groups:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        f["shared"] = {"ff": shared[0], "limit": shared[1]}
    return f


def _cfg(vocab, width, layers, eps=1e-5):
    return dict(architecture="Lomutar", vocab=vocab, width=width, norm={"eps": eps},
                layers=[{"type": "attention", "mixer": m, "mlp": f} for m, f in layers])


# a reader with a wider window than the layer it reads, one with a narrower window; groups of experts, a shared unit larger
# than the experts, limits of their own
M1 = _cfg(97, 64, [
    (_attn(4, 2, 16, 16, 8, 13, factor=3.0), _dense(96)),
    (_attn(4, 2, 16, 16, 12, 9, factor=1.5, base=500.0), _moe(32, 0.8, 12, 3, groups=(4, 2), shared=(48, 0.6))),
    (_attn(4, 2, 16, 16, 12, 30, factor=1.5, base=500.0, kv_from=1), _moe(32, 1.1, 6, 2)),
    (_attn(4, 2, 16, 16, 8, 5, factor=3.0, kv_from=0), _dense(64)),
])
# sizes that fit no vector or tile; keys and values of different widths; every query head with keys of its own; one expert a
# token; a layer without a feed-forward; a layer that sees everything, read by one with a window; no scaling; whole heads rotated
M2 = _cfg(53, 40, [
    (_attn(3, 3, 10, 6, 10, 7), None),
    (_attn(2, 1, 6, 14, 4, None, factor=2.0), _moe(18, 0.5, 5, 1, shared=(10, 1.2))),
    (_attn(4, 1, 6, 14, 4, 11, factor=2.0, kv_from=1, scale=0.3), _dense(50)),
    (_attn(3, 3, 10, 6, 10, 1), _moe(24, 2.0, 4, 4, groups=(2, 2))),
], eps=1e-3)
# widths of the tensor-core kernels: heads of 64 (tcgen05 tiles for long portions), unequal widths (windowed attention)
M3 = _cfg(200, 128, [
    (_attn(8, 1, 64, 64, 32, 70, factor=4.0, base=1e6), _moe(64, 0.7, 8, 3, groups=(4, 2), shared=(128, 0.9))),
    (_attn(4, 2, 32, 48, 16, 33, factor=2.0), _dense(256)),
    (_attn(8, 1, 64, 64, 32, 150, factor=4.0, base=1e6, kv_from=0), _moe(64, 1.3, 4, 2, groups=(2, 1))),
    (_attn(4, 2, 32, 48, 16, 20, factor=2.0, kv_from=1), _dense(64)),
])
# more query heads a kv head than a decode tile packs; heads of 128; groups of one expert each; every expert chosen
M4 = _cfg(64, 48, [
    (_attn(20, 1, 16, 16, 6, 25, factor=8.0, base=100.0), _moe(16, 0.4, 6, 2, groups=(6, 3), shared=(64, 0.4))),
    (_attn(2, 2, 128, 128, 64, 41), _moe(32, 1.0, 3, 3)),
    (_attn(2, 2, 128, 128, 64, 40, kv_from=1), _dense(32)),
])

CONFIGS = {"M1": (M1, 16), "M2": (M2, 8), "M3": (M3, 16), "M4": (M4, 4)}
LENGTHS = {"M1": [1, 2, 3, 30, 75, 41, 9, 60], "M2": [1, 5, 40, 33, 17, 64], "M3": [2, 4, 50, 240, 23, 37],
           "M4": [1, 2, 2, 19, 33, 6, 80]}


def make_tensors(cfg, seed):
    """Weights of a size that makes every mechanism matter, rounded to bfloat16 so that both precisions and the plain
    implementation hold the same numbers: gates that reach their limits on both sides, routers whose logits lie apart, sinks
    that take a good part of a short window, norm biases that do not vanish."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, spec in build_model(cfg).expected_tensors().items():
        shape = tuple(spec.shape)
        leaf = name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name
        rnd = torch.randn(shape, generator=gen)
        if name == "embed":
            t = rnd
        elif leaf in ("norm1", "final.norm"):
            t = 1.0 + rnd * 0.2
        elif leaf in ("norm1.b", "final.norm.b"):
            t = rnd * 0.3
        elif leaf == "mix.sink":
            t = rnd + 2.0
        elif len(shape) == 2:
            t = rnd * (4.0 if leaf == "mlp.router" else 1.0) / math.sqrt(shape[1])
        else:
            raise AssertionError(f"no rule for {name} {shape}")
        out[name] = t.to(torch.bfloat16).contiguous()
    return out


def make_folder(raw, seed, folder):
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(raw, f)
    save_file(make_tensors(config_from_dict(json.loads(json.dumps(raw))), seed), os.path.join(folder, "model.safetensors"))
    return folder


_cache = {}


def _setup(name, tmp_path_factory):
    if name not in _cache:
        raw, page = CONFIGS[name]
        folder = make_folder(raw, 23 + ord(name[-1]), str(tmp_path_factory.mktemp(f"lomutar{name}")))
        c, W = plain.read_config(folder), plain.read_weights(folder)
        g = torch.Generator().manual_seed(5)
        seqs = {f"r{i}": torch.randint(0, raw["vocab"], (n,), generator=g).tolist() for i, n in enumerate(LENGTHS[name])}
        ref = {rid: plain.plain_forward(c, W, toks).numpy() for rid, toks in seqs.items()}
        _cache[name] = (raw, page, folder, seqs, ref, c, W)
    return _cache[name]


def rel_err(got, ref):
    """Difference of two rows of logits, mean taken off, root mean square, over that of the reference."""
    d = np.asarray(got, dtype=np.float64) - ref
    d = d - d.mean()
    r = ref - ref.mean()
    return float(np.sqrt((d * d).mean()) / max(np.sqrt((r * r).mean()), 1e-9))


TOL = {"float32": 1e-4, "bfloat16": 0.06}
#: The share of positions that may differ by more than the tolerance, and by how much at most: a router whose scores at the
#: edge of its choice (or of its groups' choice) lie within a rounding of each other picks another expert there.
OUTLIERS = {"float32": 0.01, "bfloat16": 0.08}
OUTLIER_CAP = {"float32": 1.0, "bfloat16": 1.3}


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
    cfg = config_from_folder(make_folder(M1, 1, str(tmp_path / "m")))
    assert isinstance(cfg, LomutarConfig)
    assert config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    model = build_model(cfg)
    names = set(model.expected_tensors())
    assert {"embed", "head", "final.norm", "final.norm.b", "l0.norm1.b", "l0.mix.k", "l1.mix.sink", "l1.mlp.e11.gate",
            "l1.mlp.router", "l1.mlp.shared.down", "l2.mix.q", "l3.mlp.up"} <= names
    assert not any(n.startswith(("l2.mix.k", "l2.mix.v", "l3.mix.k", "l3.mix.v", "l2.mlp.shared")) or n.endswith("shared.sg")
                   or ".norm2" in n for n in names)
    # a plane keeps as much as the widest of the windows that read it: layer 2 reads layer 1's with a window of 30
    specs = model.kv_specs()
    assert [s.window if s is not None else None for s in specs] == [13, 30, None, None]
    assert specs[2] is None and model.entries[2].source == 1 and model.entries[3].source == 0
    open_ended = build_model(config_from_dict(json.loads(json.dumps(M2))))
    assert [s.window if s is not None else "reader" for s in open_ended.kv_specs()] == [7, None, "reader", 1]
    # one table per kind of rotation
    tables = {id(b.mixer.position) for b in model.blocks}
    assert len(tables) == 2


def test_config_errors_name_the_problem():
    def broken(change):
        raw = json.loads(json.dumps(M1))
        change(raw)
        with pytest.raises(ConfigError) as e:
            config_from_dict(raw)
        return str(e.value)

    def mixer(i):
        return lambda r: r["layers"][i]["mixer"]

    assert "layers[0].type" in broken(lambda r: r["layers"][0].update(type="gla"))
    assert "kv heads" in broken(lambda r: mixer(0)(r).update(kv_heads=3))
    assert "vdim" in broken(lambda r: mixer(0)(r).pop("vdim"))
    assert "scale" in broken(lambda r: mixer(0)(r).pop("scale"))
    assert "mask.size" in broken(lambda r: mixer(0)(r)["mask"].update(size=0))
    assert "rot.dims" in broken(lambda r: mixer(0)(r)["rot"].update(dims=18))
    assert "factor" in broken(lambda r: mixer(0)(r)["rot"].update(scaling={"factor": 0}))
    assert "kv_from" in broken(lambda r: mixer(2)(r).update(kv_from=2))
    assert "no keys and values of its own" in broken(lambda r: mixer(3)(r).update(kv_from=2))
    assert "differ" in broken(lambda r: mixer(2)(r).update(dim=32))
    assert "groups" in broken(lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(count=5))
    assert "exceeds" in broken(lambda r: r["layers"][1]["mlp"]["router"].update(top=7))
    assert "shared.limit" in broken(lambda r: r["layers"][1]["mlp"]["shared"].pop("limit"))
    assert "expert.ff" in broken(lambda r: r["layers"][1]["mlp"]["expert"].update(ff=0))
    assert "mlp.kind" in broken(lambda r: r["layers"][1]["mlp"].update(kind="sparse"))
    assert "missing keys: width" in broken(lambda r: r.pop("width"))


def test_a_missing_or_misshapen_tensor_is_named(tmp_path):
    from safetensors.torch import load_file, save_file
    from tiny_inference_server_b200.weights.loader import load_weights
    folder = make_folder(M2, 2, str(tmp_path / "m"))
    path = os.path.join(folder, "model.safetensors")
    tensors = load_file(path)
    del tensors["l0.norm1.b"]
    tensors["l1.mix.sink"] = torch.zeros(3, dtype=torch.bfloat16)
    tensors["l2.mix.k"] = torch.zeros(6, 40, dtype=torch.bfloat16)         # a layer that reads another's keys has none
    save_file(tensors, path)
    with pytest.raises(WeightError) as e:
        load_weights(folder, build_model(config_from_folder(folder)).expected_tensors())
    assert all(n in str(e.value) for n in ("l0.norm1.b", "l1.mix.sink", "l2.mix.k"))


# ------------------------------------------------------------------------------------------------
# the plain implementation against other ways of writing the same sums (CPU)
# ------------------------------------------------------------------------------------------------

def test_plain_mechanisms_written_another_way():
    g = torch.Generator().manual_seed(3)

    def rand(*s):
        return torch.randn(*s, generator=g, dtype=torch.float64)

    z, w, b = rand(5, 12) * 3 + 7, rand(12), rand(12)
    assert torch.allclose(plain.layer_norm(z, w, b, 1e-3), torch.nn.functional.layer_norm(z, (12,), w, b, 1e-3))
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    # the rotation: scores depend on the distance only; a factor stretches the positions; the rest of a head stays
    rot = {"base": 300.0, "dims": 6, "scaling": {"factor": 2.0}}
    q = rand(4, 1, 10)
    a, c = plain.rotate_pairs(q, rot, 5), plain.rotate_pairs(q, rot, 11)
    assert abs(float((a[0] * a[2]).sum() - (c[0] * c[2]).sum())) < 1e-9
    assert torch.equal(a[..., 6:], q[..., 6:])
    plain_at_3 = plain.rotate_pairs(q[:1], {"base": 300.0, "dims": 6}, 3)
    assert torch.allclose(plain.rotate_pairs(q[:1], rot, 6), plain_at_3)
    turned = torch.view_as_complex(q[0, 0, :6].reshape(3, 2).contiguous()) * torch.exp(1j * 3 * 300.0 ** (-torch.arange(3, dtype=torch.float64) / 3))
    assert torch.allclose(torch.view_as_real(turned).reshape(6), plain_at_3[0, 0, :6])
    # the softmax, key by key
    L, H, G, D, V, size = 9, 4, 2, 5, 3, 4
    qq, kk, vv, sink = rand(L, H, D), rand(L, G, D), rand(L, G, V), rand(H)
    got = plain.window_softmax(qq, kk, vv, 0.7, size, sink)
    for t in range(L):
        for h in range(H):
            den, num = math.exp(float(sink[h])), torch.zeros(V, dtype=torch.float64)
            for j in range(t + 1):
                if t - j < size:
                    e = math.exp(0.7 * float(qq[t, h] @ kk[j, h // 2]))
                    den += e
                    num += e * vv[j, h // 2]
            assert torch.allclose(got[t, h], num / den)
    # the router, expert by expert
    router = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}}
    h, Wr = rand(20, 7), rand(6, 7)
    chosen, weights = plain.route(h, Wr, router)
    two_best_differs = 0
    for t in range(20):
        s = torch.exp(h[t] @ Wr.T)
        s = (s / s.sum()).tolist()
        groups = sorted(range(3), key=lambda i: -max(s[2 * i:2 * i + 2]))[:2]
        allowed = sorted((e for e in range(6) if e // 2 in groups), key=lambda e: -s[e])[:2]
        assert chosen[t].tolist() == allowed
        assert np.allclose(weights[t].tolist(), [s[e] for e in allowed])
        two_best_differs += set(groups) != set(sorted(range(3), key=lambda i: -sum(s[2 * i:2 * i + 2]))[:2])
    assert two_best_differs > 0                                   # (the rule for a group's strength matters here)


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
    runner = make_runner(folder, "float32", 192, page_size=page, max_live=1, cuda_graphs=False, device=device)
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


def _selectors(width, parts):
    """Projections that pick columns: ``parts`` = [(name, columns)], side by side from column 0.  With them a mixer reads its
    queries, keys and values straight out of its input, so that a test can plant them."""
    W, at = {}, 0
    for name, n in parts:
        W[name] = torch.zeros(n, width, dtype=torch.float64)
        W[name][torch.arange(n), at + torch.arange(n)] = 1.0
        at += n
    return W


def _mixers(m, readers, eps, dtype, device, width):
    """The mixer of ``m`` and those of ``readers`` (configurations with ``kv_from``), loaded with projections that pick
    columns, sinks of their own and the identity as output, on one plane; (mixers, plain weights of each)."""
    from tiny_inference_server_b200.parts.base import BuildContext
    from tiny_inference_server_b200.parts.normed_attention import NormedRotaryAttention
    from tiny_inference_server_b200.parts.positions import RotaryInterleaved
    g = torch.Generator().manual_seed(m["dim"])
    ctx = BuildContext(torch.device(device), DT[dtype])
    sizes = [(x.get("mask") or {}).get("size") for x in [m] + readers]
    keep = None if any(s is None for s in sizes) else max(sizes)
    out, weights = [], []
    for x, size in zip([m] + readers, sizes):
        rot = x["rot"]
        pos = RotaryInterleaved(x["dim"], rot["base"], 512, rotary_dim=rot["dims"], factor=(rot.get("scaling") or {}).get("factor", 1.0))
        reads = x is not m
        mixer = NormedRotaryAttention(width, x["heads"], x["kv_heads"], x["dim"], x["vdim"], x["scale"], eps, pos, window=size,
                                      reads_cache=reads, cache_window=keep, prefix="")
        W = _selectors(width, [("q", x["heads"] * x["dim"]), ("k", x["kv_heads"] * x["dim"]), ("v", x["kv_heads"] * x["vdim"])])
        no = x["heads"] * x["vdim"]
        W["o"] = torch.eye(no, dtype=torch.float64)
        W["sink"] = torch.randn(x["heads"], generator=g).double()
        W["sink"][0] = 2.5
        load = dict(W, o=torch.zeros(width, no, dtype=torch.float64))
        load["o"][:no] = W["o"]
        pos.load({}, ctx)
        mixer.load({k: v.float() for k, v in load.items()}, ctx)
        out.append(mixer)
        weights.append(W)
    return out, weights


def _run_mixers(mixers, inputs, portions, page, dtype, device, pages=None):
    """Feeds ``inputs`` ({request: (L, width)}) to the mixers through a cache manager and the step layout of the engine;
    ``portions``: a list of steps, each a list of (request, rows).  The requests' slots are given back at the end.  Returns
    {request: [output of every mixer (L, columns)]} in float64."""
    from tiny_inference_server_b200.cache.manager import CacheManager
    from tiny_inference_server_b200.engine.batch import StepEntry, build_step
    from tiny_inference_server_b200.parts.base import LayerBinding
    dev = torch.device(device)
    longest = max(len(x) for x in inputs.values())
    n_pages = pages or sum((len(x) + page - 1) // page for x in inputs.values()) + 1
    cache = CacheManager([mixers[0].kv_spec()], {}, page_size=page, num_pages=n_pages, max_slots=len(inputs) + 1,
                         max_positions=longest + page, dtype=DT[dtype], device=dev, debug_poison=True)
    import random
    cache.groups[0].pool.shuffle(random.Random(1))
    grp = cache.groups[0]
    ref = cache.plane_refs[0]
    binding = LayerBinding(kv_plane=grp.plane(ref.index), kv_group=0, k_pages=grp.key_pages(ref.index), v_pages=grp.value_pages(ref.index))
    planners = []
    for mx in mixers:
        planners += [p for p in mx.step_planners() if all(p.key != q.key for q in planners)]
    fault = torch.zeros(4, dtype=torch.int32, device=dev)
    slots = {rid: cache.admit() for rid in inputs}
    fed = {rid: 0 for rid in inputs}
    out = {rid: [torch.zeros(len(x), mx.no, dtype=torch.float64) for mx in mixers] for rid, x in inputs.items()}
    for step_entries in portions:
        entries = [StepEntry(slots[rid], [0] * n, []) for rid, n in step_entries]
        starts = [cache.extend(slots[rid], n) for rid, n in step_entries]
        assert starts == [fed[rid] for rid, _ in step_entries]
        cache.sync_tables()
        step, _, _ = build_step(entries, starts, [0], [grp.table_dev], [page], fault, dev, 1, planners=planners)
        x = torch.cat([inputs[rid][fed[rid]:fed[rid] + n] for rid, n in step_entries]).to(DT[dtype]).to(dev)
        for i, mx in enumerate(mixers):
            y = mx.forward(x.clone(), step, binding).double().cpu()[:, :mx.no]
            at = 0
            for rid, n in step_entries:
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


def _planted(m, L, width, dtype, seed, window):
    """A random input of which some queries look like one key each: at the window's first place, one before it (not seen
    any more), at the sequence's first token, next to themselves, and across a page.  Query and key lie in one channel that
    is not rotated (or, where all are, the slowest one) and nowhere else, so that after the norm their score is
    ``dim * scale`` among scores of the size of ``sqrt(dim) * scale``.  Returns (input, [(query, key)])."""
    g = torch.Generator().manual_seed(seed)
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    nq, nk = H * D, G * D
    u = _round(torch.randn(L, width, generator=g), dtype)
    W = window or 10 ** 9
    pairs = []
    used = set()
    for p in (L - 1, L - 2, L - 4, L - 7, 2 * L // 3, L // 2, L // 3, L // 4, 5, 1):
        for j in (p - W + 1, p - W, 0, p - 1, p - 17):
            if 0 <= j < p and j not in used and p not in used and (window is None or not pairs or p - j >= W - 1 or len(pairs) > 3):
                pairs.append((p, j))
                used.update((p, j))
                break
    for n, (p, j) in enumerate(pairs):
        c = D - 1 - n % max(1, D - m["rot"]["dims"])
        u[p, :nq] = 0.0
        u[p, c:nq:D] = 1.5
        u[j, nq:nq + nk] = 0.0
        u[j, nq + c:nq + nk:D] = 1.5
    return u, pairs


ATTENTION_CASES = [          # heads, kv heads, dim, vdim, rotated, window, page, factor
    (4, 2, 32, 32, 16, 37, 16, 2.0),
    (8, 1, 64, 64, 32, 70, 16, 4.0),
    (2, 2, 128, 128, 64, 130, 32, 1.0),
    (6, 2, 48, 48, 24, 1, 8, 3.0),
    (6, 2, 48, 48, 24, 2, 8, 3.0),
    (3, 3, 10, 6, 4, 19, 4, 2.0),
    (4, 1, 32, 48, 16, 33, 16, 1.5),
    (20, 1, 16, 16, 8, 50, 16, 2.0),
    (12, 1, 80, 80, 8, 64, 16, 2.5),
    (4, 4, 256, 256, 128, 90, 16, 2.0),
    (4, 2, 64, 64, 32, None, 16, 8.0),
    (6, 3, 24, 40, 10, None, 5, 2.0),
    (2, 1, 64, 64, 62, 128, 64, 2.0),
]


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


def _check_attention(case, dtype, device):
    H, G, dim, vdim, rot, window, page, factor = case
    m = _attn(H, G, dim, vdim, rot, window, factor=factor, scale=14.0 / dim)
    eps = 1e-4
    width = max(H * dim + G * (dim + vdim), H * vdim)
    mixers, weights = _mixers(m, [], eps, dtype, device, width)
    L, other = 300, 90
    u, pairs = _planted(m, L, width, dtype, H * 10 + dim, window)
    b, _ = _planted(m, other, width, dtype, H * 10 + dim + 1, window)
    want = {rid: plain.attention(x, weights[0], "", m, eps)[0] for rid, x in (("a", u), ("b", b))}
    got = _run_mixers(mixers, {"a": u, "b": b}, _steps_of_two(L, other), page, dtype, device)
    tol = MECH_TOL[dtype]
    _close(got["a"][0], want["a"], tol, "attention in portions")
    _close(got["b"][0], want["b"], tol, "the request beside it")
    for p, j in pairs:
        _close(got["a"][0][p], want["a"][p], 2 * tol, f"the query at {p}, which looks for the key at {j}")
    # the planted keys matter: one key more or fewer in the window, or no sink, is far outside the tolerance
    rows = want["a"].abs().max(-1).values

    def off(changed, w=weights[0]):
        return float(((plain.attention(u, w, "", changed, eps)[0] - want["a"]).abs().max(-1).values / rows).max())
    if window:
        assert off(dict(m, mask={"size": window + 1})) > 5 * tol
        if window > 1:
            assert off(dict(m, mask={"size": window - 1})) > 5 * tol
    assert off(m, dict(weights[0], sink=torch.full((H,), -1e9, dtype=torch.float64))) > 5 * tol


@pytest.mark.parametrize("case", [c for c in ATTENTION_CASES if c[2] <= 48])
def test_attention_window_sink_and_planted_keys_cpu(case, ref_ops):
    _check_attention(case, "float32", "cpu")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ATTENTION_CASES)
def test_attention_window_sink_and_planted_keys(case, dtype):
    from tiny_inference_server_b200.kernels import ops
    before = dict(ops.calls)
    _check_attention(case, dtype, "cuda:0")
    if dtype == "bfloat16" and case[2] == case[3] and case[2] % 16 == 0 and case[0] // case[1] <= 16:
        assert ops.calls["attn_keys_rotary"] > before.get("attn_keys_rotary", 0)      # single rows: rotated in the kernel
        if case[2] in (64, 128):
            assert ops.calls["attn_tc"] > before.get("attn_tc", 0)


def _check_readers(dims, dtype, device):
    """Layers that read another layer's keys with windows wider and narrower than its own: a plane that gave pages back by
    its owner's window would show poison to the wider reader."""
    H, G, dim, vdim, page = dims
    owner = _attn(H, G, dim, vdim, dim // 2, 11, factor=2.0, scale=14.0 / dim)
    readers = [_attn(H, G, dim, vdim, dim // 2, 60, factor=2.0, scale=10.0 / dim, kv_from=0),
               _attn(H, G, dim, vdim, dim // 2, 4, factor=2.0, scale=14.0 / dim, kv_from=0)]
    eps, L = 1e-4, 200
    width = max(H * dim + G * (dim + vdim), H * vdim)
    mixers, weights = _mixers(owner, readers, eps, dtype, device, width)
    u, _ = _planted(owner, L, width, dtype, 3, 60)
    want, held = plain.attention(u, weights[0], "", owner, eps)
    wants = [want] + [plain.attention(u, w, "", m, eps, held)[0] for m, w in zip(readers, weights[1:])]
    short = _round(torch.randn(13, width, generator=torch.Generator().manual_seed(8)), dtype)
    # few pages: what falls behind the widest window is given back and used again
    pages = (60 + 40) // page + 6
    steps = [[("a", n)] for n in (40, 1, 2, 33, 1, 1, 17, 5)] + [[("b", 6), ("a", 1)], [("b", 1), ("a", 2)]] + \
        [[("a", 1)]] * 97 + [[("b", 6)]]
    got = _run_mixers(mixers, {"a": u, "b": short}, steps, page, dtype, device, pages=pages)
    for i, w in enumerate(wants):
        _close(got["a"][i], w, MECH_TOL[dtype], f"layer {i} over the shared plane")
    assert float((plain.attention(u, weights[1], "", dict(readers[0], mask={"size": 11}), eps, held)[0] - wants[1]).abs().max()) \
        > 5 * MECH_TOL[dtype] * float(wants[1].abs().max())


def test_readers_with_windows_of_their_own_cpu(ref_ops):
    _check_readers((4, 2, 16, 16, 4), "float32", "cpu")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dims", [(4, 2, 16, 16, 4), (8, 2, 64, 64, 16), (4, 1, 32, 48, 8), (3, 3, 12, 7, 4)])
def test_readers_with_windows_of_their_own(dims, dtype):
    _check_readers(dims, dtype, "cuda:0")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d", [(3, 64), (37, 40), (1, 1000), (5, 3072), (1030, 192), (2048, 1536), (1100, 30), (2, 13)])
def test_layer_norm_with_two_updates(dtype, n, d):
    """Both updates in the stream, rows whose mean is far from zero (a variance from the difference of two sums would be
    lost), few rows and many."""
    import kernel_refs
    from tiny_inference_server_b200.kernels import ops
    g = torch.Generator().manual_seed(n + d)
    res = torch.randn(n, d, generator=g) * 3
    res[n // 2] = 3000.0 + torch.randn(d, generator=g)
    da, db = (torch.randn(n, d, generator=g).to(DT[dtype]) for _ in range(2))
    w, b = 1 + 0.2 * torch.randn(d, generator=g), torch.randn(d, generator=g)
    for a1, a2 in ((da, db), (None, db), (da, None), (None, None)):
        want_res, want = res.double().clone(), torch.empty(n, d, dtype=torch.float64)
        # (the sum is what a 32-bit stream holds; the norm of it is exact)
        want_res = res.clone()
        for t in (a1, a2):
            if t is not None:
                want_res += t.float()
        z = want_res.double()
        want = plain.layer_norm(z, w.double(), b.double(), 1e-5)
        r = res.cuda()
        out = torch.empty(n, d, dtype=DT[dtype], device="cuda")
        ops.add_layer_norm(r, a1.cuda() if a1 is not None else None, a2.cuda() if a2 is not None else None, w.cuda(), b.cuda(), 1e-5, out)
        _close(r, want_res.double(), 1e-6, "the stream with its updates")
        # a row of size 3000 in 32-bit holds its deviations of size 1 to four digits
        plain_rows = torch.arange(n) != n // 2
        if plain_rows.any():
            _close(out[plain_rows.cuda()], want[plain_rows], {"float32": 1e-5, "bfloat16": 1e-2}[dtype], "layer norm")
        _close(out[n // 2], want[n // 2], {"float32": 2e-3, "bfloat16": 1e-2}[dtype], "the row far from zero")
    assert kernel_refs.add_layer_norm(res.clone(), da, db, w, b, 1e-5, torch.empty(n, d)).shape == (n, d)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("permuted", [False, True])
@pytest.mark.parametrize("H,G,dim,vdim,rot,interleaved,norm,page", [
    (4, 2, 32, 32, 16, True, True, 16), (3, 1, 96, 64, 96, True, True, 4), (2, 2, 16, 16, 6, False, True, 8),
    (5, 0, 48, 48, 20, True, True, 16), (6, 3, 128, 128, 0, True, True, 16), (2, 1, 512, 64, 256, True, True, 16),
    (2, 1, 1024, 64, 2, True, False, 16), (3, 3, 10, 6, 10, True, True, 5), (2, 1, 24, 24, 8, False, False, 3)])
def test_rotate_norm_store(dtype, permuted, H, G, dim, vdim, rot, interleaved, norm, page):
    import kernel_refs
    from tiny_inference_server_b200.kernels import ops
    if permuted and (dim % 8 or vdim % 8):
        pytest.skip("rows of whole 16-byte chunks only")
    g = torch.Generator().manual_seed(H + dim)
    n, n_pages = 21, 7
    cols = H * dim + G * (dim + vdim)
    ld = (cols + 7) // 8 * 8
    x = torch.randn(n, ld, generator=g).to(DT[dtype])
    positions = torch.tensor(list(range(3, 15)) + list(range(9)), dtype=torch.int32)
    row_slot = torch.tensor([1] * 12 + [0] * 7 + [-1] * 2, dtype=torch.int32)
    table = torch.full((2, 4 + 16 // page), -1, dtype=torch.int32)
    table[1, :(15 + page - 1) // page] = torch.randperm(n_pages, generator=g)[:(15 + page - 1) // page].to(torch.int32)
    table[0, :(7 + page - 1) // page] = torch.randperm(n_pages, generator=g)[:(7 + page - 1) // page].to(torch.int32)
    used = table[1][table[1] >= 0].tolist()
    table[0] = torch.tensor([(p if p not in used else 7 + i) if p >= 0 else -1 for i, p in enumerate(table[0].tolist())], dtype=torch.int32)
    n_pages = 7 + table.shape[1]
    cos, sin = torch.randn(40, rot // 2, generator=g), torch.randn(40, rot // 2, generator=g)
    norm_ = torch.sqrt(cos * cos + sin * sin)
    cos, sin = (cos / norm_, sin / norm_) if rot else (None, None)
    k = torch.zeros(n_pages, max(G, 1), page, dim, dtype=DT[dtype])
    v = torch.zeros(n_pages, max(G, 1), page, vdim, dtype=DT[dtype])
    xr, kr, vr, fr = x.clone(), k.clone(), v.clone(), torch.zeros(4, dtype=torch.int32)
    kernel_refs.rotate_norm_store(xr, H, G, dim, vdim, cos, sin, interleaved, norm, 1e-5, kr, vr, table, positions, row_slot, page,
                                  fr, permuted=permuted)
    xd, kd, vd, fd = x.cuda(), k.cuda(), v.cuda(), torch.zeros(4, dtype=torch.int32, device="cuda")
    ops.rotate_norm_store(xd, H, G, dim, vdim, cos.cuda() if rot else None, sin.cuda() if rot else None, interleaved, norm, 1e-5,
                          kd if G else None, vd if G else None, table.cuda(), positions.cuda(), row_slot.cuda(), page, fd,
                          permuted=permuted)
    tol = {"float32": 1e-5, "bfloat16": 1e-2}[dtype]
    _close(xd[:, :H * dim], xr[:, :H * dim].double(), tol, "queries")
    assert torch.equal(xd[:, H * dim:cols].cpu(), x[:, H * dim:cols]), "keys and values of the rows were written"
    if G:
        _close(kd, kr.double(), tol, "key rows")
        assert torch.equal(vd.cpu(), vr), "value rows"
    assert int(fd[0]) == 0


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,K,F", [(1, 64, 96), (8, 192, 320), (20, 128, 64), (30, 2048, 512), (70, 96, 64), (3100, 64, 128), (5, 40, 50),
                                   (6, 64, 20)])
def test_gated_products_in_every_form(dtype, n, K, F):
    """Product and gating (gelu, the clamped unit, silu) for every kernel that a row count goes to, with gates and up values
    well beyond the limit on both sides."""
    from tiny_inference_server_b200.kernels import ops
    from tiny_inference_server_b200.parts.base import BuildContext
    from tiny_inference_server_b200.parts.feed_forward import SwiGLU
    g = torch.Generator().manual_seed(n + F)
    x = _round(torch.randn(n, K, generator=g), dtype)
    gate, up = (_round(torch.randn(F, K, generator=g) * 2 / math.sqrt(K), dtype) for _ in range(2))
    down = _round(torch.randn(K, F, generator=g) / math.sqrt(F), dtype)
    W = {"gate": gate, "up": up, "down": down}
    wants = {"gelu": (ops.gate_gelu_tanh(), plain.gelu_gated_ff(x, W, "")),
             "clamped": (ops.gate_clamped(0.9), plain.clamped_unit(x, W, "", 0.9)),
             "silu": (None, (torch.nn.functional.silu(x @ gate.T) * (x @ up.T)) @ down.T)}
    assert float((plain.clamped_unit(x, W, "", 0.9) - plain.clamped_unit(x, W, "", 1.2)).abs().max()) > 0.1
    for name, (form, want) in wants.items():
        part = SwiGLU(K, F, names={"gate": "gate", "up": "up", "down": "down"}, stored_out_in=True, form=form)
        part.load({k: v.float() for k, v in W.items()}, BuildContext(torch.device("cuda:0"), DT[dtype]))
        _close(part.forward(x.to(DT[dtype]).cuda()), want, {"float32": 2e-5, "bfloat16": 2e-2}[dtype], name)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,d,F,E,top,groups,shared", [
    (3, 48, 40, 6, 2, (3, 2), 24), (1, 64, 96, 16, 4, (4, 1), 64), (40, 64, 32, 12, 3, (4, 2), 96), (300, 128, 64, 8, 4, None, None),
    (700, 192, 96, 16, 4, (4, 3), 96), (600, 128, 128, 8, 2, (2, 1), 192), (50, 40, 24, 5, 5, None, 16), (9, 32, 32, 4, 1, (4, 1), 32)])
def test_router_groups_and_clamped_experts(dtype, n, d, F, E, top, groups, shared):
    """The whole mixture against the plain one: few rows (a dot product per element), a hundred pairs (tiles on the tensor
    cores), a thousand (tcgen05 tiles)."""
    from tiny_inference_server_b200.kernels import ops
    from tiny_inference_server_b200.parts.base import BuildContext
    from tiny_inference_server_b200.parts.feed_forward import RoutedExperts
    g = torch.Generator().manual_seed(n + d)
    f = _moe(F, 0.7, E, top, groups=groups, shared=(shared, 1.1) if shared else None)
    gr = groups or (0, 0)
    part = RoutedExperts(d, F, E, top, gr[0], gr[1], shared or 0, scores="softmax", correction=False, group_score="best",
                         renorm=False, form=ops.gate_clamped(0.7), shared_form=ops.gate_clamped(1.1), shared_gated=False)
    W = {}
    for p in part.walk():
        for name, spec in p.expected_tensors().items():
            W[name] = _round(torch.randn(*spec.shape, generator=g) * (4.0 if name == "router" else 1.5) / math.sqrt(spec.shape[1]), dtype)
    x = _round(torch.randn(n, d, generator=g), dtype)
    want = plain.expert_mixture(x, W, "", f)
    for p in part.walk():
        p.load({k: v.float() for k, v in W.items()}, BuildContext(torch.device("cuda:0"), DT[dtype]))
    # rows whose choice hangs on a rounding are left out (there are few)
    chosen, weights = plain.route(x, W["router"], f["router"])
    noisy, _ = plain.route(x * (1 + 1e-4), W["router"] + 1e-4 * torch.randn(W["router"].shape, generator=g).double(), f["router"])
    clear = (chosen.sort(-1).values == noisy.sort(-1).values).all(-1)
    assert int(clear.sum()) >= max(1, int(0.9 * n))
    got_chosen, got_weights, _ = ops.moe_route(x.to(DT[dtype]).cuda(), part.w_router, None, None, gr[0], gr[1], top, scores="softmax",
                                               group_score="best", renorm=False)
    assert torch.equal(got_chosen.cpu().long()[clear].sort(-1).values, chosen[clear].sort(-1).values)
    _close(got_weights.cpu()[clear].sort(-1).values, weights[clear].sort(-1).values, 1e-5, "weights")
    before = dict(ops.calls)
    out = part.forward(x.to(DT[dtype]).cuda())
    _close(out[clear.cuda()], want[clear], {"float32": 2e-5, "bfloat16": 3e-2}[dtype], "mixture")
    if dtype == "bfloat16" and n * top >= 1024 and d % 64 == 0 and F % 64 == 0:
        assert ops.calls["moe_grouped_tc"] == before.get("moe_grouped_tc", 0) + 1
    elif dtype == "bfloat16" and n * top >= 96 and d % 32 == 0 and F % 32 == 0:
        assert ops.calls["moe_grouped"] == before.get("moe_grouped", 0) + 1


@gpu
def test_router_scores_far_apart_keep_their_order():
    """Scores that underflow in the softmax still choose by their logits."""
    from tiny_inference_server_b200.kernels import ops
    wr = torch.tensor([[0.0], [-300.0], [-400.0], [-200.0], [-350.0], [-500.0]])
    chosen, weights, _ = ops.moe_route(torch.ones(1, 1).cuda(), wr.cuda(), None, None, 0, 0, 3, scores="softmax", renorm=False)
    assert chosen.cpu().tolist() == [[0, 3, 1]] and weights.cpu().tolist() == [[1.0, 0.0, 0.0]]
    chosen, _, _ = ops.moe_route(torch.ones(1, 1).cuda(), wr.cuda(), None, None, 3, 1, 2, scores="softmax", group_score="best", renorm=False)
    assert chosen.cpu().tolist() == [[0, 1]]


# ------------------------------------------------------------------------------------------------
# whole models on the device
# ------------------------------------------------------------------------------------------------

@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M1", "M2", "M3", "M4"])
@pytest.mark.parametrize("mode", ["whole", "tail", "chunks", "mixed"])
def test_replay_gpu(name, mode, dtype, tmp_path, tmp_path_factory):
    raw, page, folder, seqs, ref, _, _ = _setup(name, tmp_path_factory)
    steps = _steps(mode, seqs, max_live=3)
    runner = _replay_and_compare(raw, page, folder, seqs, ref, steps, str(tmp_path / "out"), dtype, "cuda:0", TOL[dtype], max_live=3,
                                 poison=(mode == "mixed"), shuffle=(mode == "mixed"), outliers=OUTLIERS[dtype], cap=OUTLIER_CAP[dtype])
    if mode == "mixed" and name == "M1":          # its requests are long enough for the pool to turn over
        pool = runner.cache.groups[0].pool
        assert pool.allocations > pool.num_pages, "the trace does not use pages again"


@gpu
@pytest.mark.parametrize("name", ["M1", "M3"])
def test_layers_of_the_stream_gpu(name, tmp_path_factory):
    raw, page, folder, seqs, _, c, W = _setup(name, tmp_path_factory)
    _check_layers(folder, page, seqs["r5"], c, W, "cuda:0")


def random_configuration(seed):
    """A configuration drawn at random: head counts, widths, windows, rotations, readers, feed-forwards, constants."""
    import random
    rng = random.Random(seed)
    pick = rng.choice
    width = pick([24, 32, 48, 64, 96, 128, 192])
    layers, owners = [], []
    for i in range(rng.randint(2, 6)):
        if owners and rng.random() < 0.4:
            j = pick(owners)
            m = dict(json.loads(json.dumps(layers[j][0])), kv_from=j, scale=pick([0.1, 0.2, 0.4]))
            m.pop("mask", None)
        else:
            kv = pick([1, 2, 3])
            dim = pick([8, 16, 24, 32, 64, 80, 128])
            rot = pick([r for r in (2, 4, 8, 16, 24, 32, 64) if r <= dim] + [dim])
            m = _attn(kv * pick([1, 2, 3, 5]), kv, dim, pick([dim, dim, 16, 40]), rot, None, factor=pick([None, 2.0, 3.5, 8.0]),
                      base=pick([100.0, 10000.0, 1e6]))
            owners.append(i)
        size = pick([None, 1, 3, 16, 17, 40, 64, 100, 250])
        if size:
            m["mask"] = {"size": size}
        r = rng.random()
        if r < 0.1:
            mlp = None
        elif r < 0.45:
            mlp = _dense(pick([24, 32, 64, 100, 256]))
        else:
            e, top, groups = pick([(4, 1, None), (4, 2, (2, 1)), (8, 2, (4, 2)), (16, 4, (4, 3)), (6, 3, (3, 2)), (3, 3, None), (12, 2, (6, 1))])
            mlp = _moe(pick([16, 32, 64, 96]), pick([0.5, 1.0, 3.0]), e, top, groups=groups,
                       shared=pick([None, (32, 0.5), (100, 2.0), (64, 1.0)]))
        layers.append((m, mlp))
    return _cfg(rng.randint(40, 300), width, layers, eps=pick([1e-5, 1e-6, 1e-3])), pick([4, 8, 16, 16, 32])


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10])
def test_configurations_drawn_at_random(seed, dtype, tmp_path):
    """Whatever config.json says runs without a change of code: configurations drawn at random, a mixed batch of five
    requests (one of them long) through three slots over shuffled pages."""
    raw, page = random_configuration(seed)
    folder = make_folder(raw, 100 + seed, str(tmp_path / "m"))
    c, W = plain.read_config(folder), plain.read_weights(folder)
    g = torch.Generator().manual_seed(seed)
    seqs = {f"r{i}": torch.randint(0, raw["vocab"], (n,), generator=g).tolist() for i, n in enumerate([1, 2, 45, 400, 130])}
    ref = {rid: plain.plain_forward(c, W, toks).numpy() for rid, toks in seqs.items()}
    steps = trace_tools.trace_mixed(seqs, max_live=3, prefill_sizes=(64, 2, 130, 17))
    _replay_and_compare(raw, page, folder, seqs, ref, steps, str(tmp_path / "out"), dtype, "cuda:0", TOL[dtype], max_live=3,
                        poison=True, shuffle=True, outliers={"float32": 0.01, "bfloat16": 0.2}[dtype], cap=OUTLIER_CAP[dtype])


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_two_slots_used_again_and_again(dtype, tmp_path, tmp_path_factory):
    """Eight requests through two slots over poisoned pages: a page that a request reads but does not hold shows."""
    raw, page, folder, seqs, ref, _, _ = _setup("M1", tmp_path_factory)
    steps = trace_tools.trace_mixed(seqs, max_live=2, prefill_sizes=(2, 7, 3, 2), skip_every=4)
    _replay_and_compare(raw, page, folder, seqs, ref, steps, str(tmp_path / "out"), dtype, "cuda:0", TOL[dtype], max_live=2,
                        poison=True, outliers=OUTLIERS[dtype], cap=OUTLIER_CAP[dtype])


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M3", "M4"])
def test_long_decoding(name, dtype, tmp_path, tmp_path_factory):
    """A short prompt, then 300 tokens one by one, replayed from a graph: every window passes over decoded tokens only."""
    raw, page, folder, _, _, c, W = _setup(name, tmp_path_factory)
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
