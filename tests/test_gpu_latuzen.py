"""The Latuzen decoder on the GPU against the plain implementation (``plain_latuzen``): each new mechanism alone, then
whole models with random weights made here, replayed whole, token by token, in portions down to two tokens and mixed
with other requests on few pages and slots; in 32-bit and in bfloat16, eager and as captured graphs; and greedy
generation through the engine's entry point."""

from __future__ import annotations

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import plain_latuzen as plain
import traces
from latuzen_cases import CASES, attention, both, dense, memory, model, moe, own, plain_logits, random_config, random_tensors, rotation, row_error, tensor_shapes, write_folder, yarn
from test_gpu_mopilorn import check, run_trace, tokens
from test_gpu_parts import context, runtime
from test_gpu_sonalix import CUTS, as_float, bind, part_tol, rel_rows, step_mixer

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
TOL = {"float32": 1e-4, "bfloat16": 0.25}
SHARP_TOL = 1e-3
LENGTHS = {"a": [70, 3, 41, 1, 26, 97], "b": [9, 120, 33, 2, 64, 50], "c": [45, 17, 5, 80, 30], "d": [130, 20, 75, 49, 9]}


def build(tmp, name, config, seed, lengths, tokens_seed=40, change=None):
    """Two folders of one configuration: in bfloat16 the corrections alone decide which experts a token uses (rounding cannot move a
    token), in 32-bit the router follows the token.  Per storage type: folder, requests, plain logits, the logits' scale, weights."""
    out = {}
    reqs = {f"{name}{i}": tokens(config["vocab"], n, tokens_seed + i) for i, n in enumerate(lengths)}
    for dtype in ("float32", "bfloat16"):
        w = random_tensors(config, seed, fixed_choice=dtype == "bfloat16")
        if change:
            w = change(w)
        folder = write_folder(tmp / f"{name}-{dtype}", config, w)
        ref = {rid: plain_logits(config, w, t) for rid, t in reqs.items()}
        out[dtype] = (folder, reqs, ref, float(torch.cat(list(ref.values())).pow(2).mean().sqrt()), w)
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("latuzen")
    return {name: build(tmp, name, case["config"], 17 + k, LENGTHS[name]) for k, (name, case) in enumerate(sorted(CASES.items()))}


def regime_steps(reqs, regime):
    if regime == "whole":
        return traces.whole(reqs)
    if regime == "tail":
        return traces.tail_one_by_one(reqs, 40)
    if regime == "portions":
        return traces.portions(reqs)
    prompt_lens = {rid: max(1, len(t) - 14) for rid, t in reqs.items()}
    steps = traces.mixed(reqs, prompt_lens, max_live=4, seed=5)
    assert max(len(s["entries"]) for s in steps) >= 3
    return steps


# ------------------------------------------------------------------ whole models


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
@pytest.mark.parametrize("regime", ["whole", "tail", "portions", "mixed"])
def test_replay_regimes(models, name, dtype, regime):
    """Whole prompts; the last 40 tokens one by one (windows pass over decoded tokens); portions of 1 to 33 tokens;
    up to four live requests on as few pages as they need (pages and state slots are used again)."""
    folder, reqs, ref, scale, _ = models[name][dtype]
    steps = regime_steps(reqs, regime)
    outs, _ = run_trace(folder, dtype, steps, CASES[name]["block_size"])
    check(steps, outs, ref, scale, TOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
@pytest.mark.parametrize("regime", ["tail", "mixed"])
def test_replay_as_captured_graphs(models, name, dtype, regime):
    """The way generation runs by default: single-token steps and steps of more than 16 tokens as CUDA
    graphs made for padded shapes.  Padding sequences and rows must leave every cache and every state alone."""
    folder, reqs, ref, scale, _ = models[name][dtype]
    steps = traces.last_only(regime_steps(reqs, regime))
    outs, runner = run_trace(folder, dtype, steps, CASES[name]["block_size"], cuda_graphs=True)
    check(steps, outs, ref, scale, TOL[dtype])
    assert runner.core.runner.num_graph_kernels > 0


@pytest.mark.parametrize("name", ["a", "d"])
def test_batch_and_cutting_change_float32_logits_by_rounding_only(models, name):
    folder, reqs, ref, scale, _ = models[name]["float32"]
    whole, _ = run_trace(folder, "float32", traces.whole(reqs), 16)
    by_place = {}
    for rows, got in zip(traces.wanted_places(traces.whole(reqs)), whole):
        for i, place in enumerate(rows):
            by_place[place] = got[i]
    steps = regime_steps(reqs, "mixed")
    outs, _ = run_trace(folder, "float32", steps, 16)
    worst = 0.0
    for rows, got in zip(traces.wanted_places(steps), outs):
        for i, place in enumerate(rows):
            worst = max(worst, float((got[i] - by_place[place]).abs().max()))
    assert worst <= 2e-5 * scale, worst


@pytest.mark.parametrize("seed", [3, 12, 29, 41, 57, 68, 75, 90])
def test_configurations_drawn_at_random(tmp_path, seed):
    """Sizes that no hand-made case has (widths, head sizes and inner sizes that are no multiple of 8, one head, twelve heads,
    windows of a single position, pairs of dims of any count, ...), each replayed whole, in portions and mixed, in both storage types."""
    config = random_config(seed)
    block_size = [4, 8, 16, 32][seed % 4]
    made = build(tmp_path, "drawn", config, 100 + seed, [90, 1, 37, 140], tokens_seed=seed)
    for dtype, (folder, reqs, ref, scale, _) in made.items():
        for regime in ("whole", "portions", "mixed"):
            steps = regime_steps(reqs, regime) if regime != "mixed" else traces.mixed(reqs, {r: max(1, len(t) - 10) for r, t in reqs.items()}, max_live=4, seed=seed)
            outs, _ = run_trace(folder, dtype, steps, block_size)
            check(steps, outs, ref, scale, TOL[dtype])


def sharpened(w):
    """Queries and keys scaled up until a few keys take nearly all the weight (and the sink matters where none stands out)."""
    return {k: (v * 2.5).to(torch.bfloat16).float() if k.endswith(("q.norm", "k.norm")) else v for k, v in w.items()}


def test_sharp_attention_window_edges_scalings_and_shared_keys(tmp_path):
    """With sharp scores over sequences of several hundred tokens, the keys at a window's edge decide the logits: the plain model
    with a window one off, without the scaling of the frequencies (or of its pairs' size alone), with a
    layer that makes its keys anew from its own input, or with the other layout of the pairs is far outside the tolerance."""
    for name, length in (("a", 310), ("b", 260), ("c", 300)):
        case = CASES[name]
        config = case["config"]
        made = build(tmp_path, f"sharp-{name}", config, 91, [length, 110], tokens_seed=70, change=sharpened)
        folder, reqs, ref, scale, w = made["float32"]
        rid = f"sharp-{name}1"

        def worst_miss(cfg2, w2=w):
            off = plain_logits(cfg2, w2, reqs[rid])
            return max(row_error(off[i], ref[rid][i], scale) for i in range(60, 110))

        def changed(edit):
            cfg2 = json.loads(json.dumps(config))
            for ly in cfg2["layers"]:
                edit(ly, ly["mixer"] if ly["type"] == "attention" else ly["mixer"]["left"])
            return cfg2

        for d in (-1, 1):
            for kind in ("attention", "parallel"):

                def edit(ly, m):
                    if ly["type"] == kind and m["mask"]["size"] + d > 0:
                        m["mask"]["size"] += d

                assert worst_miss(changed(edit)) > 10 * SHARP_TOL, (name, kind, d)

        def halve(ly, m):  # the scaled frequencies alone
            if m["rot"].get("scaling"):
                m["rot"]["scaling"] = {**m["rot"]["scaling"], "factor": 1.0}

        assert worst_miss(changed(halve)) > 10 * SHARP_TOL, (name, "scaling")
        keep = plain.rotation_size
        plain.rotation_size = lambda rot: 1.0
        try:
            assert worst_miss(config) > 10 * SHARP_TOL, (name, "size")
        finally:
            plain.rotation_size = keep
        cfg2, w2 = json.loads(json.dumps(config)), dict(w)
        for i, ly in enumerate(cfg2["layers"]):
            j = ly["mixer"].pop("kv_from", None)
            if j is not None:
                w2.update({f"l{i}.mix.{leaf}": w[f"l{j}.mix.{leaf}"] for leaf in ("k", "v", "k.b", "v.b", "k.norm")})
        assert worst_miss(cfg2, w2) > 10 * SHARP_TOL, (name, "kv_from")
        for regime in ("whole", "tail", "portions"):
            steps = regime_steps(reqs, regime)
            outs, _ = run_trace(folder, "float32", steps, case["block_size"])
            check(steps, outs, ref, scale, SHARP_TOL, SHARP_TOL)


@pytest.mark.parametrize("name", sorted(CASES))
def test_what_would_hide_in_these_models_does_not(models, name):
    """The plain model without the sink, with a memory that forgets a little faster, with the weights renormalized
    or without the identity experts' part misses the logits by far more than the
    tolerance of the replays, wherever the model has the mechanism."""
    config = CASES[name]["config"]
    _, reqs, ref, scale, w = models[name]["float32"]
    rid = max(reqs, key=lambda r: len(reqs[r]))
    layers = config["layers"]
    routers = [ly["mlp"]["router"] for ly in layers if ly["mlp"] and ly["mlp"]["kind"] == "moe"]
    parts = {n: getattr(plain, n) for n in ("attend", "matrix_memory_walk", "route", "routed_experts")}

    def without_sink(q, k, v, s, see, sink):
        return parts["attend"](q, k, v, s, see, False)

    def forgetful(q, k, v, log_in, log_keep):
        return parts["matrix_memory_walk"](q, k, v, log_in, 1.05 * log_keep - 0.02)

    def renormalized(h, w, p, r):
        ids, wt = parts["route"](h, w, p, r)
        return ids, wt / wt.sum(-1, keepdim=True) * r["scale"]

    def no_identity(h, w, p, m):
        return parts["routed_experts"](h, {**w, **{f"{p}e{e}.{n}": torch.zeros_like(h[0]).expand(1, -1) if n != "down" else torch.zeros(h.shape[1], 1, dtype=h.dtype) for e in range(m["router"]["experts"], 99) for n in ("gate", "up", "down")}},
                                       p, {**m, "router": {**m["router"], "experts": 99}})  # fmt: skip

    wrong = []
    if any(ly["type"] == "parallel" for ly in layers):
        wrong += [("attend", without_sink), ("matrix_memory_walk", forgetful)]
    if any(r["top"] > 1 for r in routers):
        wrong.append(("route", renormalized))
    if any(r["identity"] for r in routers):
        wrong.append(("routed_experts", no_identity))
    assert wrong
    for attr, other in wrong:
        setattr(plain, attr, other)
        try:
            off = plain_logits(config, w, reqs[rid])
        finally:
            setattr(plain, attr, parts[attr])
        assert max(row_error(a, b, scale) for a, b in zip(off, ref[rid])) > 20 * TOL["float32"], attr


def test_long_decoding(models):
    """Three hundred tokens one by one after a prompt of five: windows pass over decoded tokens, their pages are given back and
    taken again, and the memories are carried through three hundred steps."""
    for name in ("a", "b", "c"):
        case = CASES[name]
        for dtype, graphs in (("float32", False), ("bfloat16", True)):
            folder, _, _, _, w = models[name][dtype]
            reqs = {"long": tokens(case["config"]["vocab"], 305, 7)}
            ref = {"long": plain_logits(case["config"], w, reqs["long"])}
            scale = float(ref["long"].pow(2).mean().sqrt())
            steps = traces.tail_one_by_one(reqs, 300)
            outs, _ = run_trace(folder, dtype, steps, case["block_size"], cuda_graphs=graphs)
            check(steps, outs, ref, scale, TOL[dtype])


def test_long_prompts_in_bfloat16(models):
    """Prompts long enough for the memory's chunked form, whole and cut so that portions of it follow single tokens and end
    inside a chunk; eager and as captured graphs (whose padding belongs to no sequence)."""
    from kvforge_b200 import ops

    for name in ("a", "c", "d"):
        case = CASES[name]
        folder, _, _, _, w = models[name]["bfloat16"]
        reqs = {"long": tokens(case["config"]["vocab"], 390, 8)}
        ref = {"long": plain_logits(case["config"], w, reqs["long"])}
        scale = float(ref["long"].pow(2).mean().sqrt())
        pos, cut = 0, []
        for n in (1, 270, 1, 2, 90, 26):
            cut.append({"step": len(cut), "entries": [{"id": "long", "tokens": reqs["long"][pos : pos + n], "want": list(range(n))}], "end": ["long"] if pos + n == 390 else []})
            pos += n
        assert pos == 390 and ops.chunks_pay(1, 270) and not ops.chunks_pay(1, 90)
        for steps in (traces.whole(reqs), cut):
            outs, _ = run_trace(folder, "bfloat16", steps, case["block_size"])
            check(steps, outs, ref, scale, TOL["bfloat16"])
            last = traces.last_only(steps)
            outs, _ = run_trace(folder, "bfloat16", last, case["block_size"], cuda_graphs=True)
            check(last, outs, ref, scale, TOL["bfloat16"])


def test_the_trace_program_reads_a_folder_and_writes_logits(models, tmp_path):
    folder, reqs, ref, scale, _ = models["b"]["float32"]
    steps = traces.portions(dict(list(reqs.items())[:3]))
    lines = "\n".join(json.dumps(s) for s in steps) + "\n"
    out = tmp_path / "out"
    res = subprocess.run(
        [sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out), "--max-tokens", "256"],
        input=lines, capture_output=True, text=True, timeout=600,
    )  # fmt: skip
    assert res.returncode == 0, res.stderr[-2000:]
    assert [ln for ln in res.stdout.splitlines() if ln.startswith("done")] == [f"done {s['step']}" for s in steps]
    vocab = CASES["b"]["config"]["vocab"]
    outs = [torch.from_numpy(np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, vocab).copy()) for s in steps]
    check(steps, outs, ref, scale, TOL["float32"])


@pytest.mark.parametrize("kind", ["attention", "parallel"])
def test_models_of_one_kind_of_mixer(tmp_path, kind):
    """A model may have layers of one kind only: attention alone keeps no state."""
    att = attention(4, 2, 16, 8, 9, rotation(12, 1000.0, yarn(2.0, 30, 4.0, 1.0) if kind == "attention" else None))
    make = (lambda ffn: own(att, ffn)) if kind == "attention" else (lambda ffn: both(att, memory(3, 12, 16, 4.0), ffn))
    config = model(77, 56, [make(dense(40)), make(None), make(moe(24, 3, 1, 2, 2, 1, 1.5))])
    for dtype, (folder, reqs, ref, scale, _) in build(tmp_path, kind, config, 7, [60, 2, 31, 85], tokens_seed=3).items():
        for regime in ("whole", "portions", "mixed"):
            steps = regime_steps(reqs, regime)
            outs, _ = run_trace(folder, dtype, steps, 8)
            check(steps, outs, ref, scale, TOL[dtype])


# ------------------------------------------------------------------ generation through the entry point


@pytest.mark.parametrize("name", sorted(CASES))
def test_greedy_generation_through_the_engine(models, name):
    """``InferenceEngine.generate`` with its scheduler: more requests than state slots, prompts cut into portions,
    decode steps as graphs, tokens read a step late."""
    from kvforge_b200 import CacheConfig, EngineConfig, InferenceEngine, SamplingParams, SchedulerConfig

    folder, _, _, _, w = models[name]["float32"]
    case = CASES[name]
    prompts = [tokens(case["config"]["vocab"], n, 300 + i) for i, n in enumerate([3, 40, 11, 1, 25, 18])]
    cfg = EngineConfig(
        cache=CacheConfig(block_size=case["block_size"], num_blocks=128),
        scheduler=SchedulerConfig(max_num_seqs=3, max_num_batched_tokens=32, max_model_len=128),
        dtype="float32",
    )
    engine = InferenceEngine(cfg, model=folder)
    outs = engine.generate(prompts, SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True))
    wd = {k: v.double() for k, v in w.items()}
    for p, o in zip(prompts, outs):
        assert o.output_token_ids == plain.greedy(case["config"], wd, p, 12)
    assert engine.core.state_slots.num_free == 3


def test_generation_from_a_named_shape():
    from kvforge_b200 import PRESETS, EngineConfig, InferenceEngine, SamplingParams, SchedulerConfig

    cfg = EngineConfig(model=PRESETS["latuzen-tiny"], scheduler=SchedulerConfig(max_num_seqs=4, max_num_batched_tokens=64, max_model_len=256), dtype="bfloat16")
    outs = InferenceEngine(cfg).generate([[1, 2, 3], list(range(40))], SamplingParams(max_tokens=8, temperature=0.0, ignore_eos=True))
    assert all(len(o.output_token_ids) == 8 for o in outs)


# ------------------------------------------------------------------ mechanisms alone


def rounded(shapes, dtype, seed, gain=1.5):
    """Random tensors by local name: norm weights around one, biases small, matrices of unit gain times ``gain``."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for k, s in shapes.items():
        r = torch.randn(s, generator=g)
        t = 1.0 + 0.2 * r if k.endswith(("norm", "out")) else 2.0 + 2.0 * r if k.endswith("f.b") else 0.3 * r if k.endswith(".b") else r * gain / s[-1] ** 0.5
        out[k] = t.to(dtype).float()
    return out


def mixer_of(config, layer):
    """The layer's mixer as the model's description builds it, and its tensors' shapes by their names under the mixer."""
    from kvforge_b200.config.latuzen_config import LatuzenConfig
    from kvforge_b200.models.latuzen import latuzen_spec
    from kvforge_b200.parts.base import build_part

    prefix = f"l{layer}.mix."
    part = build_part("mixer", latuzen_spec(LatuzenConfig.from_dict(config)).layers[layer].block.params["mixer"], prefix)
    return part, {k[len(prefix) :]: s for k, s in tensor_shapes(config).items() if k.startswith(prefix)}


def pages(nb, nkv, bs, dk, dv, dtype):
    from kvforge_b200.parts.base import LayerCache

    up = lambda n: (n + 7) // 8 * 8  # noqa: E731
    return LayerCache(torch.zeros(nb, nkv, bs, up(dk), device="cuda", dtype=dtype), torch.zeros(nb, nkv, bs, up(dv), device="cuda", dtype=dtype), 0)


ROT = {"whole": (1.0, None), "part": (0.5, yarn(4.0, 40, 6.0, 1.0)), "scaled": (1.0, yarn(8.0, 20, 4.0, 0.5))}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [1, 7, 33, 64, 400])
@pytest.mark.parametrize("nh,nkv,dk,dv,t,bs,turns", [(6, 3, 24, 16, 45, 4, "part"), (3, 1, 10, 13, 60, 8, "scaled"), (8, 2, 64, 64, 200, 16, "part"), (9, 3, 64, 64, 150, 16, "scaled"),
                                                     (4, 2, 128, 128, 150, 16, "whole"), (2, 2, 6, 40, 50, 4, "part")])  # fmt: skip
def test_attention_with_joint_norms_that_turns(dtype, window, nh, nkv, dk, dv, t, bs, turns):
    """The whole sequence in one step, then portions and single tokens on top of the cache, against the plain mixer; heads of 64 and
    of 128 on pages of 16 go to the tensor-core kernels in bfloat16.  A second layer reads the first one's cache with queries
    and a longer window of its own, and writes nothing."""
    width, eps = 80, 1e-5
    part_of, scaling = ROT[turns]
    rot = rotation(max(2, int(dk * part_of) // 2 * 2), 500.0, scaling)
    config = model(50, width, [own(attention(nh, nkv, dk, dv, window, rot), None), own(attention(nkv, nkv, dk, dv, window + 20, rot, scale=0.3, kv_from=0), None)], eps)
    rt = runtime(dtype)
    made, ws = [], []
    for layer in (0, 1):
        part, shapes = mixer_of(config, layer)
        w = rounded(shapes, dtype, 3 + layer)
        bind(part, w, dtype, rt)
        made.append(part)
        ws.append({"m." + k: v.double() for k, v in w.items()})
    m, m2 = (ly["mixer"] for ly in config["layers"])
    g = torch.Generator().manual_seed(5)
    x, x2 = (torch.randn(t, width, generator=g).to(dtype) for _ in range(2))
    k, v = plain.keys_and_values(x.double(), ws[0], "m.", m, eps)
    ref = plain.jointly_normed_attention(x.double(), ws[0], "m.", m, eps, k, v)
    ref2 = plain.jointly_normed_attention(x2.double(), ws[1], "m.", m2, eps, k, v)
    table = [int(i) for i in torch.randperm(64, generator=g)]
    need = made[0].cache_need()
    assert (need.kind, need.window) == ("window", window + 20)
    for cuts in CUTS(t):
        cache = pages(64, nkv, bs, dk, dv, dtype)
        got = step_mixer(made[0], rt, x, bs, table, cuts, cache)
        assert rel_rows(got, ref) < part_tol(dtype), cuts
        before = cache.k.clone()
        cache.writable = False
        got = step_mixer(made[1], rt, x2, bs, table, cuts, cache)
        assert rel_rows(got, ref2) < part_tol(dtype), (cuts, "shared")
        assert torch.equal(before, cache.k)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("interleaved", [False, True])
def test_joint_norm_turns_either_layout(dtype, interleaved):
    """The kernel alone: both layouts of the pairs, rotations of all and of a part of a head (counts that do and do not go four numbers a
    thread), with and without the norm, rows of the storage type and slices of a split product."""
    from kvforge_b200 import ops

    g = torch.Generator().manual_seed(3)
    n, nh, nkv = 5, 3, 2
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")  # noqa: E731
    pos = [0, 1, 17, 300, 2]
    for dk, dv, dims in ((16, 8, 16), (16, 12, 12), (16, 8, 6), (10, 6, 10), (12, 8, 2), (24, 8, 0)):
        for norm in (True, False):
            for sliced in (False, True):
                width = nh * dk + nkv * (dk + dv) + 8
                rows = torch.randn(3, n, width, generator=g)
                y = rows.sum(0).to(dtype) if not sliced else torch.zeros(n, width, dtype=dtype)
                src = rows.sum(0).double() if sliced else y.double()
                qw, kw = 1.0 + 0.2 * torch.randn(nh * dk, generator=g), 1.0 + 0.2 * torch.randn(nkv * dk, generator=g)
                rot = rotation(max(dims, 2), 100.0, yarn(4.0, 20, 4.0, 1.0))
                kc, vc = (torch.zeros(4, nkv, 4, d, dtype=dtype, device="cuda") for d in (dk, dv))
                slots = [3, 5, 9, 1, 14]
                out = y.cuda()
                ops.joint_norm_cache(
                    out, ops.Partials(rows.cuda()) if sliced else None, None, qw.cuda() if norm else None, kw.cuda() if norm else None, nh * dk, nkv * dk, 1e-5,
                    i32(slots), kc, vc, nh, nkv, dk, dv, 4, positions=i32(pos), inv_freq=torch.tensor(plain.frequencies(rot)).float().cuda() if dims else None,
                    interleaved=interleaved, magnitude=plain.rotation_size(rot) if dims else 1.0,
                )  # fmt: skip
                q, k = src[:, : nh * dk], src[:, nh * dk : (nh + nkv) * dk]
                if norm:
                    q, k = plain.unit_rms(q, 1e-5) * qw.double(), plain.unit_rms(k, 1e-5) * kw.double()

                def turned(z, heads):
                    z = z.reshape(n, heads, dk)
                    if not dims:
                        return z
                    every = torch.zeros(max(pos) + 1, heads, dk, dtype=torch.float64)
                    every[pos] = z
                    return plain.rotate(every, rot, interleaved)[pos]

                tol = 2e-4 if dtype == torch.float32 else 3e-2
                assert rel_rows(out[:, : nh * dk].float().cpu(), turned(q, nh).reshape(n, -1)) < tol, (dk, dims, norm, sliced)
                keys = torch.stack([kc[s // 4, :, s % 4] for s in slots]).float().cpu()
                assert rel_rows(keys, turned(k, nkv)) < tol, (dk, dims, norm, sliced)
                values = torch.stack([vc[s // 4, :, s % 4] for s in slots]).float().cpu()
                assert rel_rows(values, src[:, (nh + nkv) * dk : (nh + nkv) * dk + nkv * dv].reshape(n, nkv, dv)) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [1, 9, 64, 400])
@pytest.mark.parametrize("nh,nkv,dk,dv,t,bs,dims", [(6, 3, 24, 16, 45, 4, 24), (3, 1, 10, 13, 60, 8, 6), (8, 2, 64, 64, 200, 16, 16), (4, 2, 128, 128, 150, 16, 128), (8, 4, 64, 40, 90, 16, 64)])
def test_attention_with_normed_heads_and_a_sink_of_score_zero(dtype, window, nh, nkv, dk, dv, t, bs, dims):
    """The left side of a parallel mixer alone; heads whose size is no multiple of 8 are padded."""
    from kvforge_b200.config.latuzen_config import LatuzenConfig
    from kvforge_b200.models.latuzen import _left
    from kvforge_b200.parts.base import build_part

    width, eps = 80, 1e-5
    m = attention(nh, nkv, dk, dv, window, rotation(dims, 500.0), scale=0.2)
    config = model(50, width, [both(m, memory(1, 4, 4, 1.0), None)], eps)
    cfg = LatuzenConfig.from_dict(config)
    rt = runtime(dtype)
    part = build_part("mixer", _left(cfg, cfg.layers[0].mixer.left), "m.")
    w = rounded({k[len("l0.mix.left.") :]: s for k, s in tensor_shapes(config).items() if k.startswith("l0.mix.left.") and not k.endswith(".out")}, dtype, 3)
    bind(part, w, dtype, rt)
    g = torch.Generator().manual_seed(5)
    x = torch.randn(t, width, generator=g).to(dtype)
    wd = {"m." + k: v.double() for k, v in w.items()}
    ref = plain.sink_attention(x.double(), wd, "m.", m, eps)
    table = [int(i) for i in torch.randperm(64, generator=g)]
    for cuts in CUTS(t):
        got = step_mixer(part, rt, x, bs, table, cuts, pages(64, nkv, bs, dk, dv, dtype))
        assert rel_rows(got, ref) < part_tol(dtype), cuts


@pytest.mark.parametrize("side", ["joint", "left"])
def test_one_far_key_and_keys_at_a_window_edge(side):
    """A query that matches one key and nothing else (that one score stands out): far back, at the sequence's first places, around
    borders of pages, of key tiles and of the decode form's key ranges, and just inside and just outside the query's window; in
    a prompt and decoded.  The rotation turns dims that hold zeros, so that distance does not move the score."""
    from kvforge_b200.config.latuzen_config import LatuzenConfig
    from kvforge_b200.models.latuzen import _left
    from kvforge_b200.parts.base import build_part

    width, nh, nkv, dk, dv, bs, eps, t = 32, 2, 1, 64, 64, 16, 1e-6, 300
    for dtype in (torch.float32, torch.bfloat16):
        rt = runtime(dtype, max_tokens=512)
        for window in (300, 200, 129, 27):
            edge = t - window
            for far in sorted({0, 1, 15, 16, 63, 64, 127, 128, 255, 256, max(0, edge - 1), edge, edge + 1, t - 2}):
                g = torch.Generator().manual_seed(far)
                m = attention(nh, nkv, dk, dv, window, rotation(16, 500.0), scale=0.4 if side == "left" else 1.0)
                config = model(50, width, [own(m, None) if side == "joint" else both(m, memory(1, 4, 4, 1.0), None)], eps)
                if side == "joint":
                    part, shapes = mixer_of(config, 0)
                else:
                    cfg = LatuzenConfig.from_dict(config)
                    part = build_part("mixer", _left(cfg, cfg.layers[0].mixer.left), "m.")
                    shapes = {k[len("l0.mix.left.") :]: s for k, s in tensor_shapes(config).items() if k.startswith("l0.mix.left.") and not k.endswith(".out")}
                w = rounded(shapes, dtype, 9)
                w = {k: torch.zeros_like(v) if k in ("q", "k") or k.endswith(".b") else torch.ones_like(v) if k.endswith("norm") else v for k, v in w.items()}
                # the queries read the input's first number, the keys its second (and a constant third, so that all are of one size)
                for h in range(nh):
                    w["q"][h * dk + 40, 0] = 1.0
                w["k"][40, 1] = 1.0
                w["k"][41, 2] = 1.0
                x = 0.5 * torch.randn(t, width, generator=g)
                x[:, 0], x[:, 1], x[:, 2] = 1.0, 0.0, 1.0
                x[far, 1], x[far, 2] = 1.0, 0.0
                x = x.to(dtype)
                bind(part, w, dtype, rt)
                wd = {"m." + k: v.double() for k, v in w.items()}

                def plain_mixer(z):
                    if side == "left":
                        return plain.sink_attention(z, wd, "m.", m, eps)
                    return plain.jointly_normed_attention(z, wd, "m.", m, eps, *plain.keys_and_values(z, wd, "m.", m, eps))

                ref = plain_mixer(x.double())
                x_off = x.double()
                x_off[far, 1], x_off[far, 2] = 0.0, 1.0
                assert (rel_rows(plain_mixer(x_off)[-1:], ref[-1:]) > 0.2) == (far >= edge), (window, far)  # the key is seen, and then it is all there is
                table = [int(i) for i in torch.randperm(32, generator=g)]
                for cuts in ([(0, t)], [(0, t - 1), (t - 1, t)], [(0, 150), (150, t - 2), (t - 2, t)]):
                    got = step_mixer(part, rt, x, bs, table, cuts, pages(32, nkv, bs, dk, dv, dtype))
                    assert rel_rows(got[-1:], ref[-1:]) < (1e-4 if dtype == torch.float32 else 3e-2), (window, far, cuts)


def memory_part(width, m, eps):
    from kvforge_b200.parts.base import PartSpec, build_part

    h, dk, dv = m["heads"], m["dim"], m["vdim"]
    part = build_part("mixer", PartSpec("matrix_memory", {"hidden_size": width, "num_heads": h, "head_dim": dk, "v_head_dim": dv, "gate_cap": m["gate_cap"], "eps": eps}), "m.")
    shapes = {"q": (h * dk, width), "k": (h * dk, width), "v": (h * dv, width), "g": (h * dv, width), "o": (width, h * dv), "norm": (h * dv,),
              "i": (h, width), "i.b": (h,), "f": (h, width), "f.b": (h,)}  # fmt: skip
    return part, shapes


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dk,dv,cap,t", [(2, 16, 24, 15.0, 45), (3, 10, 6, 0.7, 60), (1, 32, 12, 4.0, 50), (2, 128, 64, 15.0, 150), (4, 64, 128, 8.0, 90), (2, 9, 5, 30.0, 40), (16, 32, 31, 15.0, 60), (1, 300, 8, 15.0, 45)])
def test_matrix_memory_through_the_state(dtype, heads, dk, dv, cap, t):
    """Whole, in portions and token by token; in a slot that another request has used; beside another request."""
    from kvforge_b200.parts.base import LayerCache

    rt = runtime(dtype)
    width, eps = 72, 1e-6
    m = memory(heads, dk, dv, cap)
    part, shapes = memory_part(width, m, eps)
    w = rounded(shapes, dtype, 7)
    bind(part, w, dtype, rt)
    assert part.cache_need().kind == "none"
    g = torch.Generator().manual_seed(8)
    x, x2 = torch.randn(t, width, generator=g).to(dtype), torch.randn(23, width, generator=g).to(dtype)
    wd = {"m." + k: v.double() for k, v in w.items()}
    ref, ref2 = (plain.matrix_memory(v.double(), wd, "m.", m, eps) for v in (x, x2))
    cache = LayerCache(None, None, -1, True, torch.zeros(4, *part.state_shape(), device="cuda"))
    tol = 1e-4 if dtype == torch.float32 else 8e-2  # a head whose sums cancel is divided by a small number
    mean = lambda a, b: float((a.double() - b.double()).abs().mean() / b.double().abs().mean())  # noqa: E731
    for cuts in CUTS(t):
        cache.state[2] = 0  # the slot was used by the run before: a new request starts from zero
        got = step_mixer(part, rt, x, 1024, [0], cuts, cache, slot=2)
        assert rel_rows(got, ref) < tol and mean(got, ref) < tol / 4, cuts
    # the second half of one request beside the whole of another, in slots of their own; other slots stay zero
    n2, half = x2.shape[0], t // 2
    cache.state.zero_()
    ctx = context(rt, [half], [0], 4, [[0]], [0] * half)
    ctx.state_slots = torch.tensor([3], dtype=torch.int32, device="cuda")
    part.forward(ctx, x[:half].cuda(), cache)
    ctx = context(rt, [n2, t - half], [0, half], 4, [[0], [0]], [0] * (n2 + t - half))
    ctx.state_slots = torch.tensor([1, 3], dtype=torch.int32, device="cuda")
    got = as_float(part.forward(ctx, torch.cat([x2, x[half:]]).cuda(), cache), n2 + t - half).cpu()
    assert rel_rows(got[:n2], ref2) < tol and rel_rows(got[n2:], ref[half:]) < tol
    assert float(cache.state[0].abs().max()) == 0.0 and float(cache.state[2].abs().max()) == 0.0


def run_memory(q, k, v, zi, zf, bi, bf, cap, parts, slots, state_rows, chunked):
    """The recurrence's kernels on several sequences over several steps (``parts``: rows of each sequence in each step); the read-out divided
    and undivided by hand, and the states."""
    from kvforge_b200 import ops

    i32 = lambda z: torch.tensor(z, dtype=torch.int32, device="cuda")  # noqa: E731
    n, h, dk = q.shape
    dv = v.shape[2]
    dvx = ops.memory_columns(dv)
    floats = h * dk * dvx + h
    state = torch.zeros(state_rows, floats + (-floats % 4) + 4, device="cuda")
    view = state[:, 4 : 4 + floats]
    lens = [sum(p[i] for p in parts) for i in range(len(slots))]
    starts = [sum(lens[:i]) for i in range(len(lens))]
    got, done = torch.zeros(n, h, dv), [0] * len(lens)
    zpad = -(-h // 8) * 8
    for part in parts:
        idx = [s0 + d + j for s0, d, m in zip(starts, done, part) for j in range(m)]
        qsl = [0]
        for m in part:
            qsl.append(qsl[-1] + m)
        rows = len(idx)
        x = torch.cat([q[idx].reshape(rows, -1), k[idx].reshape(rows, -1), v[idx].reshape(rows, -1)], dim=1).cuda()
        z = torch.zeros(rows, 2 * zpad)
        z[:, :h], z[:, zpad : zpad + h] = zi[idx], zf[idx]
        out, floor = torch.full((rows, h * dvx), float("nan"), device="cuda"), torch.full((rows, h), float("nan"), device="cuda")
        raw = torch.full((rows, h * ops.CHUNK_TOKENS), float("nan"), device="cuda") if chunked else None
        ops.matrix_memory(x, 0, h * dk, 2 * h * dk, dk**-0.5, z.cuda(), zpad, bi.cuda(), bf.cuda(), cap, view, out, floor, i32(qsl), i32(slots), len(slots), h, dk, dv,
                          max_query_len=max(part), raw=raw)  # fmt: skip
        o = out.cpu().reshape(rows, h, dvx).double()
        got[idx] = (o[..., :dv] / (torch.maximum(o[..., dv].abs(), floor.cpu().double()) + 1e-6)[..., None]).float()
        done = [d + m for d, m in zip(done, part)]
    return got, state, starts, lens


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("heads,dk,dv,cap", [(4, 16, 24, 15.0), (3, 4, 3, 2.0), (2, 128, 100, 15.0), (5, 100, 36, 8.0), (16, 64, 128, 15.0)])
def test_memory_kernels_with_gates_of_every_size(chunked, heads, dk, dv, cap):
    """The kernels in 32-bit against the plain walk: sequences of 1 to 300 tokens side by side (chunks that are full, end early or hold one
    token), states carried from step to step at places that are no chunk's edge, forget gates from none at all to ones
    that leave nothing of the past, input gates from far below the floor (where e^(-m) is the divisor) to ones that outweigh
    everything before them, a slot of no sequence left alone."""
    g = torch.Generator().manual_seed(heads + dk)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    parts = [[200, 1, 30, 64, 2], [100, 0, 100, 0, 65]]
    n = sum(map(sum, parts))
    q, k, v = r(n, heads, dk), r(n, heads, dk), r(n, heads, dv)
    bi, bf = 4.0 * r(heads), torch.tensor([[30.0, 6.0, 2.0, 0.0, -30.0][h % 5] for h in range(heads)])
    zi, zf = 3.0 * r(n, heads), 2.0 * r(n, heads)
    zi[::11] += 12.0  # now and then a token that outweighs the past
    zi[5::13] -= 30.0
    zf[::17] -= 40.0  # and a step that forgets everything
    got, state, starts, lens = run_memory(q, k, v, zi, zf, bi, bf, cap, parts, [5, 0, 3, 6, 1], 7, chunked)
    li, lf = cap * torch.tanh((zi + bi).double() / cap), plain.log_sigmoid(cap * torch.tanh((zf + bf).double() / cap))
    for rid, (s0, m) in enumerate(zip(starts, lens)):
        rows = slice(s0, s0 + m)
        ref = plain.matrix_memory_walk(q[rows].double() * dk**-0.5, k[rows].double(), v[rows].double(), li[rows], lf[rows])
        # a divisor near the floor of the read-out's cancellation makes single numbers large: measure against each one's size
        err = (got[rows].double() - ref).abs() / (1.0 + ref.abs())
        assert float(err.max()) < 2e-3 and float(err.mean()) < 2e-5, rid
        assert rel_rows(got[rows], ref) < 5e-4, rid
    assert float(state[[2, 4]].abs().max()) == 0.0 and float(state[:, :4].abs().max()) == 0.0


def test_memory_state_is_the_same_bits_however_it_is_cut():
    g = torch.Generator().manual_seed(5)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    heads, dk, dv, n = 3, 20, 12, 97
    args = (r(n, heads, dk), r(n, heads, dk), r(n, heads, dv), 3 * r(n, heads), 2 + 2 * r(n, heads), r(heads), r(heads), 15.0)
    whole, s0, _, _ = run_memory(*args, [[n]], [1], 2, False)
    for parts in ([[1]] * n, [[40], [1], [2], [54]]):
        got, s1, _, _ = run_memory(*args, parts, [1], 2, False)
        assert torch.equal(got, whole) and torch.equal(s0, s1)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [1, 9, 40])
@pytest.mark.parametrize("into_stream", [False, True])
def test_attention_beside_a_memory(dtype, n, into_stream):
    """Both branches behind one input product, their normed mean as a result or added to the float stream; then the following
    token on what they left."""
    from kvforge_b200 import ops

    for left, right in ((attention(4, 2, 16, 24, 7, rotation(8, 100.0)), memory(2, 16, 8, 15.0)), (attention(3, 1, 12, 20, 50, rotation(12, 100.0)), memory(3, 10, 5, 2.0))):
        rt = runtime(dtype)
        width, bs = 56, 4
        config = model(50, width, [both(left, right, None)], eps=1e-5)
        part, shapes = mixer_of(config, 0)
        w = rounded(shapes, dtype, 21)
        for branch, name in zip(part.sub_parts(), ("left.", "right.")):
            bind(branch, {k[len(name) :]: v for k, v in w.items() if k.startswith(name)}, dtype, rt)
        bind(part, w, dtype, rt)
        assert part.open
        x = torch.randn(n + 1, width, generator=torch.Generator().manual_seed(2)).to(dtype)
        ref = plain.side_by_side(x.double(), {"m." + k: v.double() for k, v in w.items()}, "m.", {"left": left, "right": right}, 1e-5)
        cache = pages(32, left["kv_heads"], bs, left["dim"], left["vdim"], dtype)
        cache.state = torch.zeros(2, *part.state_shape(), device="cuda")
        table = list(range(31, -1, -1))
        got = []
        for a, b in ((0, n), (n, n + 1)):
            ctx = context(rt, [b - a], [a], bs, [table], [table[p // bs] * bs + p % bs for p in range(a, b)])
            ctx.state_slots = torch.tensor([1], dtype=torch.int32, device="cuda")
            if into_stream:
                ctx.residual = torch.full((b - a, width), 2.0, device="cuda")
                assert part.forward(ctx, x[a:b].cuda(), cache) is ops.ADDED
                got.append(ctx.residual.cpu() - 2.0)
            else:
                got.append(as_float(part.forward(ctx, x[a:b].cuda(), cache), b - a).cpu().clone())
        assert rel_rows(torch.cat(got), ref) < (1e-4 if dtype == torch.float32 else 6e-2)
        assert float(cache.state[0].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_router_with_groups_ranked_by_their_best_member(dtype):
    """Softmax scores, corrections (negative ones among them) that move the choice alone, groups ranked by their largest corrected
    score, scaled weights; for one token and for many."""
    from kvforge_b200 import ops

    g = torch.Generator().manual_seed(3)
    differs = 0
    for n, width, choices, top, groups, keep, scale in ((1, 64, 8, 2, 4, 2, 2.5), (7, 50, 12, 3, 3, 1, 0.5), (300, 96, 40, 4, 8, 3, 1.0), (9, 64, 6, 1, 6, 2, 3.0), (33, 40, 9, 9, 3, 3, 1.5)):
        x, router = torch.randn(n, width, generator=g).to(dtype), torch.randn(choices, width, generator=g) / width**0.5
        correction = 0.3 * torch.randn(choices, generator=g) - 0.2
        ids, wts = torch.zeros(n, top, dtype=torch.int32, device="cuda"), torch.zeros(n, top, device="cuda")
        args = (x.cuda(), router.cuda(), correction.cuda(), top, groups, keep, 0.0, ids, wts, True, False)
        ops.moe_route(*args, group_rank="max", scale=scale)
        r = {"top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}
        want, weights = plain.route(x.double(), {"router": router.double(), "correction": correction.double()}, "", r)
        assert ids.tolist() == want
        assert torch.allclose(wts.cpu().double(), weights, rtol=1e-5, atol=1e-7)
        ops.moe_route(*args)
        differs += int(ids.tolist() != want)
    assert differs  # on some of these inputs the sum of a group's two best would choose otherwise


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [1, 5, 40, 400])
@pytest.mark.parametrize("ff,experts,identity,top", [(64, 4, 2, 2), (30, 3, 5, 3), (48, 2, 0, 1), (40, 1, 3, 2)])
def test_experts_that_hand_their_input_on(dtype, n, ff, experts, identity, top):
    """The feed-forward part against the plain one, for one token, a few and many (from 64 rows an expert on average the products
    run on the tcgen05 tensor cores, whose rows of identity pairs hold nothing); steps in which no token uses a real expert."""
    from kvforge_b200 import ops
    from kvforge_b200.parts.base import PartSpec, build_part

    rt = runtime(dtype, max_tokens=512)
    width, choices, scale = 48, experts + identity, 1.7
    part = build_part("ffn", PartSpec("routed_experts", {
        "hidden_size": width, "experts": experts, "identity": identity, "top": top, "intermediate_size": ff, "correction": True, "score": "softmax",
        "normalize": False, "weight_scale": scale, "group_rank": "max", "activation": "gated"}), "m.")  # fmt: skip
    for only_identity in (False, True):
        if only_identity and identity < top:
            continue
        g = torch.Generator().manual_seed(11)
        w = {"router": torch.randn(choices, width, generator=g) * 0.1, "correction": torch.randn(choices, generator=g)}
        if only_identity:
            w["correction"][experts:] += 10.0
        for e in range(experts):
            for name, rows, cols in (("gate", ff, width), ("up", ff, width), ("down", width, ff)):
                w[f"e{e}.{name}"] = (torch.randn(rows, cols, generator=g) * 0.3).to(dtype).float()
        bind(part, w, dtype, rt)
        x = torch.randn(n, width, generator=g).to(dtype)
        r = {"experts": experts, "identity": identity, "top": top, "groups": {"count": 1, "keep": 1}, "scale": scale}
        ref = plain.routed_experts(x.double(), {"m." + k: v.double() for k, v in w.items()}, "m.", {"router": r})
        # rows of the pairs of identity experts are never written: whatever lies there must not show
        for buf in rt._buffers.values():
            if buf.is_floating_point():
                buf.fill_(float("nan"))
        ctx = context(rt, [n], [0], 4, [[0]], [0] * n)
        got = as_float(part.forward(ctx, x.cuda()), n).cpu()
        assert rel_rows(got, ref) < part_tol(dtype)
        resid = torch.ones(n, width, device="cuda")
        ctx.residual = resid
        assert part.forward(ctx, x.cuda()) is ops.ADDED
        assert rel_rows(resid.cpu() - 1.0, ref) < part_tol(dtype) + 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layer_norm_with_a_bias(dtype):
    """On the stream plus what is pending (a tensor, slices, nothing); rows gathered before the head; widths that do and do not take
    four numbers a thread, and one beyond the form that keeps rows in registers."""
    from kvforge_b200 import ops
    from kvforge_b200.parts.base import PartSpec, build_part

    rt = runtime(dtype)
    g = torch.Generator().manual_seed(2)
    for width in (64, 100, 37, 2048, 4100):
        part = build_part("norm", PartSpec("layernorm", {"dim": width, "eps": 1e-5, "bias": True, "names": {"weight": "n", "bias": "n.b"}}), "x.")
        assert sorted(part.tensor_name(k) for k in type(part).weight_decls(part.params)) == ["x.n", "x.n.b"]
        w, b = 1.0 + 0.2 * torch.randn(width, generator=g), torch.randn(width, generator=g)
        part.bind({"weight": w.cuda(), "bias": b.cuda()}, rt)
        n = 7
        stream = 3.0 + torch.randn(n, width, generator=g)
        y, slices = torch.randn(n, width, generator=g).to(dtype), torch.randn(13, n, width, generator=g)
        for pending, add in ((None, 0.0), (y.cuda(), y.double()), (ops.Partials(slices.cuda()), slices.double().sum(0))):
            resid = stream.cuda()
            total = stream.double() + add
            got = part.forward(None, resid, pending)
            assert rel_rows(got.float().cpu(), plain.layer_norm(total, w.double(), b.double(), 1e-5)) < part_tol(dtype)
            assert rel_rows(resid.cpu(), total) < 1e-6
            rows = torch.tensor([5, 0, 5], dtype=torch.int32, device="cuda")
            got = part.forward(None, stream.cuda(), pending, rows=rows, num_rows=3)
            assert rel_rows(got.float().cpu(), plain.layer_norm(total, w.double(), b.double(), 1e-5)[[5, 0, 5]]) < part_tol(dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [1, 3, 16, 17, 100, 200])
def test_a_parallel_layer_hands_on_the_slices_of_both_parts(dtype, n):
    """A layer whose two output products both run over slices of K (few tokens: the decode product; some dozens: the library's): the
    slices come as one set; with more tokens, and in 32-bit, the results are added otherwise.  The sum is the plain layer's."""
    from kvforge_b200 import ops
    from kvforge_b200.config.latuzen_config import LatuzenConfig
    from kvforge_b200.models.latuzen import latuzen_spec
    from kvforge_b200.parts.base import build_part

    width, bs = 128, 16
    m = attention(32, 2, 64, 64, 40, rotation(64, 500.0))
    config = model(50, width, [own(m, dense(2048))])
    rt = runtime(dtype)
    block = build_part("block", latuzen_spec(LatuzenConfig.from_dict(config)).layers[0].block, "l0.")
    w = rounded({k: s for k, s in tensor_shapes(config).items() if k.startswith("l0.")}, dtype, 4)
    w = {k: 1.0 + 0.2 * v if k == "l0.norm1" else v for k, v in w.items()}
    for part in block.sub_parts():
        own_w = {local: w[part.tensor_name(local)] for local in type(part).weight_decls(part.params)}
        part.params = {**part.params, "names": {}}
        bind(part, own_w, dtype, rt)
    stream = torch.randn(n, width, generator=torch.Generator().manual_seed(1))
    wd = {k: v.double() for k, v in w.items()}
    h = plain.layer_norm(stream.double(), wd["l0.norm1"], wd["l0.norm1.b"], 1e-6)
    want = plain.jointly_normed_attention(h, wd, "l0.mix.", m, 1e-6, *plain.keys_and_values(h, wd, "l0.mix.", m, 1e-6)) + plain.feed_forward(h, wd, "l0.mlp.", config["layers"][0]["mlp"])
    ctx = context(rt, [n], [0], bs, [list(range(16))], list(range(n)))
    resid = stream.cuda()
    ctx.residual = resid
    left = block.forward(ctx, resid, None, pages(16, 2, bs, 64, 64, dtype))
    if dtype == torch.bfloat16 and n <= 128:
        assert isinstance(left, ops.Partials) and left.nsplit >= 4 and torch.equal(resid.cpu(), stream)
    assert ctx.slices is None
    got = resid.cpu().double() - stream.double()
    if left is not ops.ADDED:
        got = got + as_float(left, n).cpu().double()
    assert rel_rows(got, want) < part_tol(dtype)


@pytest.mark.parametrize("d", [64, 128])
@pytest.mark.parametrize("nh,nkv,window,lens", [(8, 2, 0, [150, 3, 70]), (4, 4, 40, [90, 1, 33, 129]), (16, 2, 70, [700, 20])])
def test_learned_sinks_on_the_tensor_core_kernels(d, nh, nkv, window, lens):
    """Sinks of every size (far below every score to far above) as the tcgen05 kernel takes them for prompts and the TMA kernel for
    decoding, its ranges merged through the scratch, through a cluster, or a single one."""
    from kvforge_b200 import ops

    g = torch.Generator().manual_seed(d + nh)
    bs, scale, dev = 16, d**-0.5, "cuda"
    i32 = lambda z: torch.tensor(z, dtype=torch.int32, device=dev)  # noqa: E731
    sinks = torch.tensor([[-50.0, 0.0, 1.5, 3.0, 20.0][h % 5] for h in range(nh)])
    n = sum(lens)
    q, k, v = (1.5 * torch.randn(n, h, d, generator=g).bfloat16() for h in (nh, nkv, nkv))
    per = -(-max(lens) // bs)
    tables = torch.randperm(len(lens) * per, generator=g).reshape(len(lens), per)
    kc, vc = (torch.zeros(len(lens) * per, nkv, bs, d, dtype=torch.bfloat16) for _ in range(2))
    want, at = torch.zeros(n, nh, d, dtype=torch.float64), 0
    for b, m in enumerate(lens):
        rows = slice(at, at + m)
        for p in range(m):
            kc[tables[b, p // bs], :, p % bs], vc[tables[b, p // bs], :, p % bs] = k[at + p], v[at + p]
        see = plain.window_mask(m, window or m)
        for h in range(nh):
            s = (q[rows, h].double() @ k[rows, h // (nh // nkv)].double().T * scale).masked_fill(~see, float("-inf"))
            p = torch.softmax(torch.cat([s, torch.full((m, 1), float(sinks[h]), dtype=torch.float64)], dim=1), dim=1)[:, :m]
            want[rows, h] = p @ v[rows, h // (nh // nkv)].double()
        at += m
    qsl = i32([0] + [sum(lens[: i + 1]) for i in range(len(lens))])
    args = (kc.cuda(), vc.cuda(), tables.int().cuda())
    err = torch.zeros(1, dtype=torch.int32, device=dev)
    out = torch.zeros(n, nh * d, dtype=torch.bfloat16, device=dev)
    ops.paged_attention(q.reshape(n, -1).cuda(), out, *args, qsl, i32(lens), len(lens), max(lens), nh, nkv, d, scale, window=window, err=err, sinks=sinks.cuda(), kernel="tcgen05")
    assert int(err) == 0
    assert rel_rows(out.float().cpu(), want.reshape(n, -1)) < 2e-2
    last = [sum(lens[: i + 1]) - 1 for i in range(len(lens))]
    for split, cluster in ((64, False), (64, True), (1024, False), (1024, True)):
        b = len(lens)
        sa, sm = ops.attention_scratch_shapes(b, nh, d, max(lens), split)
        scratch = (torch.empty(sa, device=dev), torch.empty(sm, device=dev), torch.zeros(b * nkv, dtype=torch.int32, device=dev))
        out = torch.zeros(b, nh * d, dtype=torch.bfloat16, device=dev)
        ops.paged_attention(q[last].reshape(b, -1).cuda(), out, *args, i32(list(range(b + 1))), i32(lens), b, 1, nh, nkv, d, scale, window=window, err=err, sinks=sinks.cuda(),
                            scratch=scratch, max_context=max(lens), split_size=split, cluster=cluster, kernel="tma")  # fmt: skip
        assert int(err) == 0
        assert rel_rows(out.float().cpu(), want[last].reshape(b, -1)) < 2e-2, (split, cluster)
