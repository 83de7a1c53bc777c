"""The Ritizen decoder on the GPU against the plain implementation (``plain_ritizen``): each new mechanism alone, then
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

import plain_ritizen as plain
import traces
from ritizen_cases import CASES, attention, lightning, mamba2, parallel, plain_logits, random_config, random_tensors, row_error, write_folder
from test_gpu_mopilorn import check, run_trace, tokens
from test_gpu_parts import context, runtime
from test_gpu_sonalix import CUTS, as_float, bind, part_tol, rel_rows, step_mixer

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
TOL = {"float32": 1e-4, "bfloat16": 0.25}
SHARP_TOL = 1e-3
LENGTHS = {"a": [70, 3, 41, 1, 26, 97], "b": [9, 120, 33, 2, 64, 50], "c": [45, 17, 5, 80, 30], "d": [130, 20, 75, 49, 9], "e": [61, 14, 2, 90, 27]}


def build(tmp, name, config, w, lengths, seed=40):
    folder = write_folder(tmp / name, config, w)
    reqs = {f"{name}{i}": tokens(config["vocab"], n, seed + i) for i, n in enumerate(lengths)}
    ref = {rid: plain_logits(config, w, t) for rid, t in reqs.items()}
    scale = float(torch.cat(list(ref.values())).pow(2).mean().sqrt())
    return folder, reqs, ref, scale, w


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """Per case: folder, requests, plain logits of every request whole, the logits' scale, weights."""
    tmp = tmp_path_factory.mktemp("ritizen")
    return {name: build(tmp, name, case["config"], random_tensors(case["config"], 17 + k), LENGTHS[name]) for k, (name, case) in enumerate(sorted(CASES.items()))}


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
    """Whole prompts; the last 40 tokens one by one (chunks begin and end among decoded tokens); portions of 1 to 33 tokens;
    up to four live requests on as few pages as they need (pages and state slots are used again)."""
    folder, reqs, ref, scale, _ = models[name]
    steps = regime_steps(reqs, regime)
    outs, _ = run_trace(folder, dtype, steps, CASES[name]["block_size"])
    check(steps, outs, ref, scale, TOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
@pytest.mark.parametrize("regime", ["tail", "mixed"])
def test_replay_as_captured_graphs(models, name, dtype, regime):
    """The way generation runs by default: single-token steps and steps of more than 16 tokens as CUDA
    graphs made for padded shapes.  Padding sequences and rows must leave every cache and every state alone."""
    folder, reqs, ref, scale, _ = models[name]
    steps = traces.last_only(regime_steps(reqs, regime))
    outs, runner = run_trace(folder, dtype, steps, CASES[name]["block_size"], cuda_graphs=True)
    check(steps, outs, ref, scale, TOL[dtype])
    assert runner.core.runner.num_graph_kernels > 0


@pytest.mark.parametrize("name", ["a", "d"])
def test_batch_and_cutting_change_float32_logits_by_rounding_only(models, name):
    folder, reqs, ref, scale, _ = models[name]
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
    chunks of a single position, six taps, ...), each replayed whole, in portions and mixed, in both storage types."""
    config = random_config(seed)
    block_size = [4, 8, 16, 32][seed % 4]
    folder, reqs, ref, scale, _ = build(tmp_path, "drawn", config, random_tensors(config, 100 + seed), [90, 1, 37, 140], seed=seed)
    for dtype in ("float32", "bfloat16"):
        for regime in ("whole", "portions", "mixed"):
            steps = regime_steps(reqs, regime) if regime != "mixed" else traces.mixed(reqs, {r: max(1, len(t) - 10) for r, t in reqs.items()}, max_live=4, seed=seed)
            outs, _ = run_trace(folder, dtype, steps, block_size)
            check(steps, outs, ref, scale, TOL[dtype])


def sharpened(w):
    """Queries and keys scaled up until a few keys take nearly all the weight."""
    return {k: (v * 3.0).to(torch.bfloat16).float() if k.endswith(("q.norm", "k.norm")) else v for k, v in w.items()}


def test_sharp_attention_far_keys_chunk_edges_gates_and_shared_keys(tmp_path):
    """With sharp scores over sequences of several hundred tokens, a far key among hundreds and the keys at a chunk's edge decide
    the logits: the plain model with a chunk one off, without positions, with a layer that makes its keys anew from its
    own input, or with its states cut off at a place is far outside the tolerance."""
    for name, length in (("a", 310), ("b", 300), ("c", 310), ("e", 220)):
        case = CASES[name]
        config = case["config"]
        w = sharpened(random_tensors(config, seed=91))
        folder, reqs, ref, scale, _ = build(tmp_path, f"sharp-{name}", config, w, [length, 150], seed=70)
        rid = f"sharp-{name}1"

        def worst_miss(cfg2, w2):
            off = plain_logits(cfg2, w2, reqs[rid])
            return max(row_error(off[i], ref[rid][i], scale) for i in range(60, 150))

        chunked = [i for i, ly in enumerate(config["layers"]) if ly["type"] == "parallel" and ly["mixer"]["left_scale"] != 0.0]
        for d in (-1, 1):
            if chunked:
                cfg2 = json.loads(json.dumps(config))
                for i in chunked:
                    cfg2["layers"][i]["mixer"]["left"]["mask"]["size"] += d
                assert worst_miss(cfg2, w) > 10 * SHARP_TOL, (name, "chunk", d)
        shared = [i for i, ly in enumerate(config["layers"]) if ly["mixer"].get("kv_from") is not None]
        if shared:
            cfg2, w2 = json.loads(json.dumps(config)), dict(w)
            for i in shared:
                j = cfg2["layers"][i]["mixer"].pop("kv_from")
                p = f"l{j}.mix." if config["layers"][j]["type"] == "attention" else f"l{j}.mix.left."
                for leaf in ("k", "v", "k.norm"):
                    w2[f"l{i}.mix.{leaf}"] = w[p + leaf]
            assert worst_miss(cfg2, w2) > 10 * SHARP_TOL, (name, "kv_from")
        assert worst_miss(config, dict(w, pos=0 * w["pos"])) > 10 * SHARP_TOL, (name, "pos")
        for regime in ("whole", "tail", "portions"):
            steps = regime_steps(reqs, regime)
            outs, _ = run_trace(folder, "float32", steps, case["block_size"])
            check(steps, outs, ref, scale, SHARP_TOL, SHARP_TOL)


def test_long_decoding(models):
    """Three hundred tokens one by one after a prompt of five: chunks begin many times among decoded tokens, their pages are given
    back and taken again, and the states are carried through three hundred steps."""
    for name in ("a", "b", "e"):
        case = CASES[name]
        folder, _, _, _, w = models[name]
        reqs = {"long": tokens(case["config"]["vocab"], 305, 7)}
        ref = {"long": plain_logits(case["config"], w, reqs["long"])}
        scale = float(ref["long"].pow(2).mean().sqrt())
        steps = traces.tail_one_by_one(reqs, 300)
        for dtype, graphs in (("float32", False), ("bfloat16", True)):
            outs, _ = run_trace(folder, dtype, steps, case["block_size"], cuda_graphs=graphs)
            check(steps, outs, ref, scale, TOL[dtype])


def test_long_prompts_in_bfloat16(models):
    """Prompts long enough for the recurrences' chunked form, whole and cut so that portions of it follow single tokens and end
    inside a chunk; eager and as captured graphs (whose padding belongs to no sequence)."""
    from kvforge_b200 import ops

    for name in ("a", "d", "e"):
        case = CASES[name]
        folder, _, _, _, w = models[name]
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
    folder, reqs, ref, scale, _ = models["b"]
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


@pytest.mark.parametrize("kind", ["attention", "parallel", "mamba2"])
def test_models_of_one_kind_of_mixer(tmp_path, kind):
    """A model may have layers of one kind only: state spaces alone keep no pages at all (state slots only), attention alone no
    state."""
    from ritizen_cases import layer, model

    mixer = {"attention": attention(4, 2, 16, 8), "parallel": parallel(attention(2, 1, 16, 8, chunk=9), lightning(3, 12, 16, [0.9, 0.97, 0.5])),
             "mamba2": mamba2(4, 16, 24, 2, norm_groups=2)}[kind]  # fmt: skip
    config = model(77, 56, [layer(kind, mixer, 40), layer(kind, mixer, None)], max_positions=100)
    folder, reqs, ref, scale, w = build(tmp_path, kind, config, random_tensors(config, 7), [60, 2, 31, 85], seed=3)
    for dtype in ("float32", "bfloat16"):
        for regime in ("whole", "portions", "mixed"):
            steps = regime_steps(reqs, regime)
            outs, _ = run_trace(folder, dtype, steps, 8)
            check(steps, outs, ref, scale, TOL[dtype])
    if kind == "mamba2":
        from kvforge_b200 import EngineConfig, InferenceEngine, SamplingParams, SchedulerConfig

        engine = InferenceEngine(EngineConfig(scheduler=SchedulerConfig(max_num_seqs=2, max_num_batched_tokens=16, max_model_len=64), dtype="float32"), model=folder)
        prompts = [tokens(77, n, 9 + n) for n in (5, 20, 1)]
        outs = engine.generate(prompts, SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True))
        wd = {k: v.double() for k, v in w.items()}
        for p, o in zip(prompts, outs):
            assert o.output_token_ids == plain.greedy(config, wd, p, 6)


# ------------------------------------------------------------------ generation through the entry point


@pytest.mark.parametrize("name", ["a", "b", "d", "e"])
def test_greedy_generation_through_the_engine(models, name):
    """``InferenceEngine.generate`` with its scheduler: more requests than state slots, prompts cut into portions,
    decode steps as graphs, tokens read a step late."""
    from kvforge_b200 import CacheConfig, EngineConfig, InferenceEngine, SamplingParams, SchedulerConfig

    folder, _, _, _, w = models[name]
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


def test_generation_from_a_named_shape_and_the_longest_sequence():
    """The named tiny shape with random weights; a request that would pass the table of positions is not admitted."""
    from kvforge_b200 import PRESETS, EngineConfig, InferenceEngine, SamplingParams, SchedulerConfig

    cfg = EngineConfig(model=PRESETS["ritizen-tiny"], scheduler=SchedulerConfig(max_num_seqs=4, max_num_batched_tokens=64, max_model_len=4096), dtype="bfloat16")
    assert cfg.scheduler.max_model_len == PRESETS["ritizen-tiny"].max_position_embeddings
    engine = InferenceEngine(cfg)
    outs = engine.generate([[1, 2, 3], list(range(40))], SamplingParams(max_tokens=8, temperature=0.0, ignore_eos=True))
    assert all(len(o.output_token_ids) == 8 for o in outs)


# ------------------------------------------------------------------ mechanisms alone


def rounded(shapes, dtype, seed, gain=1.5):
    """Random tensors by local name: norm weights around one, biases small, matrices of unit gain times ``gain``."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for k, s in shapes.items():
        r = torch.randn(s, generator=g)
        t = 1.0 + 0.2 * r if k.endswith("norm") or k == "D" else 0.7 * r - 1.0 if k in ("A_log", "dt_bias") else 0.3 * r if k.endswith(".b") or k == "conv" else r * gain / s[-1] ** 0.5
        out[k] = t.to(dtype).float()
    return out


def attention_part(width, m, eps, gate="head", bias=False, shared=False):
    from kvforge_b200.parts.base import PartSpec, build_part

    return build_part("mixer", PartSpec("gated_attention", {
        "hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"], "scale": m["scale"],
        "chunk": (m.get("mask") or {}).get("size"), "qkv_bias": bias, "joint_norm": {"eps": eps}, "gate": gate, "shared_kv": shared}), "m.")  # fmt: skip


def attention_shapes(width, m, gate, bias, shared=False):
    h, g, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rows = {"q": h * dk} if shared else {"q": h * dk, "k": g * dk, "v": g * dv}
    out = {n: (r, width) for n, r in rows.items()}
    out.update({f"{n}.b": (r,) for n, r in rows.items() if bias})
    out.update({f"{n}.norm": (r,) for n, r in rows.items() if n != "v"})
    return {**out, "g": (h if gate == "head" else h * dv, width), "o": (width, h * dv)}


def pages(nb, nkv, bs, dk, dv, dtype):
    from kvforge_b200.parts.base import LayerCache

    up = lambda n: (n + 7) // 8 * 8  # noqa: E731
    return LayerCache(torch.zeros(nb, nkv, bs, up(dk), device="cuda", dtype=dtype), torch.zeros(nb, nkv, bs, up(dv), device="cuda", dtype=dtype), 0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("chunk", [None, 1, 7, 33, 64, 70])
@pytest.mark.parametrize("nh,nkv,dk,dv,t,bs", [(6, 3, 24, 16, 45, 4), (3, 1, 9, 13, 60, 8), (8, 2, 64, 64, 200, 16), (9, 3, 64, 64, 150, 16), (4, 2, 128, 128, 150, 16), (2, 2, 16, 40, 50, 4)])
def test_attention_with_joint_norms_gates_and_chunks(dtype, chunk, nh, nkv, dk, dv, t, bs):
    """One gate a head without biases, and one a channel with them; the whole sequence in one step, then portions and single
    tokens on top of the cache, against the plain mixer; heads of 64 and of 128 on pages of 16 go to the tensor-core
    kernels in bfloat16.  A second layer reads the first one's cache with queries of its own, and writes nothing."""
    width, eps = 80, 1e-5
    for gate, bias in (("head", False), ("channel", True)):
        rt = runtime(dtype)
        m = attention(nh, nkv, dk, dv, chunk=chunk)
        part, w = attention_part(width, m, eps, gate, bias), rounded(attention_shapes(width, m, gate, bias), dtype, 3)
        bind(part, w, dtype, rt)
        m2 = attention(nkv, nkv, dk, dv, scale=0.3)
        reader, w2 = attention_part(width, m2, eps, shared=True), rounded(attention_shapes(width, m2, "head", False, shared=True), dtype, 4)
        bind(reader, w2, dtype, rt)
        g = torch.Generator().manual_seed(5)
        x, x2 = (torch.randn(t, width, generator=g).to(dtype) for _ in range(2))
        wd, wd2 = ({"m." + k: v.double() for k, v in ws.items()} for ws in (w, w2))
        k, v = plain.keys_and_values(x.double(), wd, "m.", m, eps)
        ref = plain.attention(x.double(), wd, "m.", m, eps, k, v)
        ref2 = plain.attention(x2.double(), wd2, "m.", m2, eps, k, v)
        table = [int(i) for i in torch.randperm(64, generator=g)]
        need = part.cache_need()
        assert (need.kind, need.window) == (("chunk", chunk) if chunk else ("full", None))
        for cuts in CUTS(t):
            cache = pages(64, nkv, bs, dk, dv, dtype)
            got = step_mixer(part, rt, x, bs, table, cuts, cache)
            assert rel_rows(got, ref) < part_tol(dtype), (cuts, gate)
            before = cache.k.clone()
            cache.writable = False
            got = step_mixer(reader, rt, x2, bs, table, cuts, cache)
            assert rel_rows(got, ref2) < part_tol(dtype), (cuts, "shared")
            assert torch.equal(before, cache.k)


def test_one_far_key_and_keys_at_a_chunk_edge():
    """A query that matches one key and nothing else (that one score stands out): far back, at the sequence's first places, around
    borders of pages, of key tiles and of the decode form's key ranges, and just inside and just outside the query's chunk; in
    a prompt and decoded."""
    width, nh, nkv, dk, dv, bs, eps, t = 32, 2, 1, 64, 64, 16, 1e-6, 300
    for dtype in (torch.float32, torch.bfloat16):
        rt = runtime(dtype, max_tokens=512)
        for chunk in (None, 100, 150, 27):
            first = 0 if chunk is None else (t - 1) // chunk * chunk
            for far in sorted({0, 1, 15, 16, 63, 64, 127, 128, 255, 256, max(0, first - 1), first, first + 1, t - 2}):
                g = torch.Generator().manual_seed(far)
                m = attention(nh, nkv, dk, dv, scale=1.0, chunk=chunk)
                w = rounded(attention_shapes(width, m, "head", False), dtype, 9)
                w.update({"q": torch.zeros(nh * dk, width), "k": torch.zeros(nkv * dk, width), "q.norm": torch.ones(nh * dk), "k.norm": torch.ones(nkv * dk)})
                # the queries read the input's first number, the keys its second (and a constant third, so that all are of one size)
                for h in range(nh):
                    w["q"][h * dk, 0] = 1.0
                w["k"][0, 1] = 1.0
                w["k"][1, 2] = 1.0
                x = 0.5 * torch.randn(t, width, generator=g)
                x[:, 0], x[:, 1], x[:, 2] = 1.0, 0.0, 1.0
                x[far, 1], x[far, 2] = 1.0, 0.0
                x = x.to(dtype)
                part = attention_part(width, m, eps)
                bind(part, w, dtype, rt)
                wd = {"m." + k: v.double() for k, v in w.items()}
                xd = x.double()
                ref = plain.attention(xd, wd, "m.", m, eps, *plain.keys_and_values(xd, wd, "m.", m, eps))
                x_off = xd.clone()
                x_off[far, 1], x_off[far, 2] = 0.0, 1.0
                off = plain.attention(x_off, wd, "m.", m, eps, *plain.keys_and_values(x_off, wd, "m.", m, eps))
                assert (rel_rows(off[-1:], ref[-1:]) > 0.2) == (far >= first), (chunk, far)  # the key is seen, and then it is all there is
                table = [int(i) for i in torch.randperm(32, generator=g)]
                for cuts in ([(0, t)], [(0, t - 1), (t - 1, t)], [(0, 150), (150, t - 2), (t - 2, t)]):
                    got = step_mixer(part, rt, x, bs, table, cuts, pages(32, nkv, bs, dk, dv, dtype))
                    assert rel_rows(got[-1:], ref[-1:]) < (1e-4 if dtype == torch.float32 else 3e-2), (chunk, far, cuts)


def two_requests(part, rt, x, ref, x2, ref2, cache, dtype):
    """The second half of one request beside the whole of another, in slots of their own; other slots stay zero."""
    t, n2 = x.shape[0], x2.shape[0]
    cache.state.zero_()
    half = t // 2
    ctx = context(rt, [half], [0], 4, [[0]], [0] * half)
    ctx.state_slots = torch.tensor([3], dtype=torch.int32, device="cuda")
    part.forward(ctx, x[:half].cuda(), cache)
    ctx = context(rt, [n2, t - half], [0, half], 4, [[0], [0]], [0] * (n2 + t - half))
    ctx.state_slots = torch.tensor([1, 3], dtype=torch.int32, device="cuda")
    got = as_float(part.forward(ctx, torch.cat([x2, x[half:]]).cuda(), cache), n2 + t - half).cpu()
    assert rel_rows(got[:n2], ref2) < part_tol(dtype)
    assert rel_rows(got[n2:], ref[half:]) < part_tol(dtype)
    assert float(cache.state[0].abs().max()) == 0.0 and float(cache.state[2].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dv,n,groups,taps,parts,t", [(4, 16, 24, 2, 4, 2, 60), (3, 7, 5, 1, 5, 3, 45), (6, 8, 16, 3, 2, 1, 50), (2, 24, 40, 1, 1, 4, 40), (8, 64, 128, 2, 4, 2, 150),
                                                            (1, 12, 33, 1, 3, 1, 40), (16, 32, 64, 1, 4, 1, 90), (2, 5, 300, 2, 6, 1, 40)])  # fmt: skip
def test_state_space_through_the_state(dtype, heads, dv, n, groups, taps, parts, t):
    """Whole, in portions and token by token; in a slot that another request has used; beside another request."""
    from kvforge_b200.parts.base import LayerCache, PartSpec, build_part

    rt = runtime(dtype)
    width, eps = 72, 1e-6
    m = mamba2(heads, dv, n, groups, conv=taps, norm_groups=parts)
    part = build_part("mixer", PartSpec("state_space", {"hidden_size": width, "num_heads": heads, "v_head_dim": dv, "state_dim": n, "groups": groups, "conv": taps, "norm_groups": parts, "eps": eps}), "m.")
    inner, gn = heads * dv, groups * n
    shapes = {"in": (2 * inner + 2 * gn + heads, width), "conv": (inner + 2 * gn, taps), "conv.b": (inner + 2 * gn,), "dt_bias": (heads,), "A_log": (heads,), "D": (heads,), "norm": (inner,), "o": (width, inner)}
    w = rounded(shapes, dtype, 7)
    bind(part, w, dtype, rt)
    assert part.cache_need().kind == "none"
    g = torch.Generator().manual_seed(8)
    x, x2 = torch.randn(t, width, generator=g).to(dtype), torch.randn(23, width, generator=g).to(dtype)
    wd = {"m." + k: v.double() for k, v in w.items()}
    ref, ref2 = (plain.mamba2(v.double(), wd, "m.", m, eps) for v in (x, x2))
    cache = LayerCache(None, None, -1, True, torch.zeros(4, *part.state_shape(), device="cuda"))
    for cuts in CUTS(t):
        cache.state[2] = 0  # the slot was used by the run before: a new request starts from zero
        got = step_mixer(part, rt, x, 1024, [0], cuts, cache, slot=2)
        assert rel_rows(got, ref) < part_tol(dtype), cuts
    two_requests(part, rt, x, ref, x2, ref2, cache, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dk,dv,t", [(2, 16, 24, 45), (3, 10, 6, 60), (1, 32, 12, 50), (2, 128, 64, 150), (4, 64, 128, 90), (2, 9, 5, 40)])
def test_lightning_attention_through_the_state(dtype, heads, dk, dv, t):
    """Retention with silu on its projections, one norm over all heads and a logistic gate; as above."""
    from kvforge_b200.parts.base import LayerCache, PartSpec, build_part

    rt = runtime(dtype)
    width, eps = 72, 1e-6
    decay = [[0.9, 0.99, 0.9375, 1.0][h % 4] for h in range(heads)]
    m = lightning(heads, dk, dv, decay)
    part = build_part("mixer", PartSpec("retention", {"hidden_size": width, "num_heads": heads, "head_dim": dk, "v_head_dim": dv, "decay": decay, "eps": eps, "key_scale": 1.0,
                                                      "activation": "silu", "norm": "joint", "gate": "sigmoid"}), "m.")  # fmt: skip
    shapes = {"q": (heads * dk, width), "k": (heads * dk, width), "v": (heads * dv, width), "g": (heads * dv, width), "o": (width, heads * dv), "norm": (heads * dv,)}
    w = rounded(shapes, dtype, 7)
    bind(part, w, dtype, rt)
    g = torch.Generator().manual_seed(8)
    x, x2 = torch.randn(t, width, generator=g).to(dtype), torch.randn(23, width, generator=g).to(dtype)
    wd = {"m." + k: v.double() for k, v in w.items()}
    ref, ref2 = (plain.lightning_attention(v.double(), wd, "m.", m, eps) for v in (x, x2))
    cache = LayerCache(None, None, -1, True, torch.zeros(4, heads * dk * dv, device="cuda"))
    for cuts in CUTS(t):
        cache.state[2] = 0
        got = step_mixer(part, rt, x, 1024, [0], cuts, cache, slot=2)
        assert rel_rows(got, ref) < part_tol(dtype), cuts
    two_requests(part, rt, x, ref, x2, ref2, cache, dtype)


@pytest.mark.parametrize("per_token", [False, True])
@pytest.mark.parametrize("heads,groups,dk,dv", [(4, 4, 16, 24), (6, 2, 20, 12), (3, 1, 4, 4), (2, 2, 128, 100), (8, 1, 128, 64), (5, 5, 100, 36), (40, 2, 64, 128)])
def test_recurrences_chunk_by_chunk(per_token, heads, groups, dk, dv):
    """The chunked form in 32-bit against the plain walks: sequences of 1 to 300 tokens side by side (chunks that are full, end early
    or hold one token), states carried from step to step at places that are no chunk's edge, decays from none at all to ones
    that leave nothing of a token's past, a slot of no sequence left alone."""
    from kvforge_b200 import ops

    if not per_token and groups != heads:
        pytest.skip("heads with a fixed decay have keys of their own")
    g = torch.Generator().manual_seed(heads + dk)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")  # noqa: E731
    lens, parts = [300, 1, 130, 64, 67], [[200, 1, 30, 64, 2], [100, 0, 100, 0, 65]]
    n = sum(lens)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    q, k, v = r(n, groups, dk), r(n, groups, dk) / dk**0.5, r(n, heads, dv)
    starts = [sum(lens[:i]) for i in range(len(lens))]
    decay = torch.tensor([[1.0, 0.9995, 0.9, 0.5, 1e-6][h % 5] for h in range(heads)])
    a_log, bias = 1.5 * r(heads), r(heads)
    dt = 2.0 * r(n, heads)
    dt[::7] += 12.0  # now and then a step that forgets everything
    ref = torch.zeros(n, heads, dv, dtype=torch.float64)
    for s0, m in zip(starts, lens):
        rows = slice(s0, s0 + m)
        if per_token:
            d = plain.softplus(dt[rows].double() + bias.double())
            ref[rows] = plain.state_space_walk(v[rows].double(), k[rows].double(), q[rows].double(), d, a_log.double(), torch.zeros(heads, dtype=torch.float64))
        else:
            ref[rows] = plain.fixed_decay_walk(q[rows].double(), k[rows].double(), v[rows].double(), decay.double().tolist())
    state = torch.zeros(7, heads * dk * dv + 4, device="cuda")
    view = state[:, 4:]
    slots = [5, 0, 3, 6, 1]
    got = torch.zeros(n, heads, dv)
    done = [0] * len(lens)
    for part in parts:
        idx = [s0 + d + j for s0, d, m in zip(starts, done, part) for j in range(m)]
        qsl = [0]
        for m in part:
            qsl.append(qsl[-1] + m)
        rows, out = len(idx), torch.full((len(idx), heads * dv), float("nan"), device="cuda")
        raw = torch.full((rows, groups * ops.CHUNK_TOKENS), float("nan"), device="cuda")
        if per_token:
            x = torch.cat([v[idx].reshape(rows, -1), k[idx].reshape(rows, -1), q[idx].reshape(rows, -1)], dim=1).cuda()
            ops.state_space(x, dt[idx].cuda(), bias.cuda(), a_log.cuda(), view, out, i32(qsl), i32(slots), len(lens), heads, groups, dk, dv, max_query_len=max(part), raw=raw)
        else:
            x = torch.cat([q[idx].reshape(rows, -1), k[idx].reshape(rows, -1), v[idx].reshape(rows, -1)], dim=1).cuda()
            ops.retention(x, 0, heads * dk, 2 * heads * dk, i32([0] * rows), None, False, 1.0, decay.cuda(), view, out, i32(qsl), i32(slots), len(lens), heads, dk, dv,
                          max_query_len=max(part), log_decay=decay.double().log().float().cuda(), raw=raw)  # fmt: skip
        got[idx] = out.cpu().reshape(rows, heads, dv)
        done = [d + m for d, m in zip(done, part)]
    assert rel_rows(got, ref) < 2e-5
    for rid, (s0, m) in enumerate(zip(starts, lens)):
        assert rel_rows(got[s0 : s0 + m], ref[s0 : s0 + m]) < 5e-5, rid
    assert float(state[[2, 4]].abs().max()) == 0.0 and float(state[:, :4].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_wide_norm_and_gate(dtype):
    """Parts and the whole row, the gate before and after the norm, with and without what passes the recurrence by, a constant,
    rows that do and do not take four numbers a thread, results into part of a wider row."""
    from kvforge_b200 import ops

    g = torch.Generator().manual_seed(1)
    for c, heads, parts in ((48, 4, 2), (35, 5, 1), (36, 4, 6), (2560, 8, 1), (33, 3, 3)):
        n = 9
        o, w, d = torch.randn(n, c, generator=g), 1.0 + 0.2 * torch.randn(c, generator=g), torch.randn(heads, generator=g)
        x, z = (torch.randn(n, c, generator=g).to(dtype) for _ in range(2))
        for act, first, skip, mult in (("silu", True, True, 1.0), ("sigmoid", False, False, -0.7), (None, False, True, 0.0), ("sigmoid", True, False, 1.3), ("silu", False, True, 0.5)):
            u = o.double() + (d.double().repeat_interleave(c // heads) * x.double() if skip else 0.0)
            a = 1.0 if act is None else plain.silu(z.double()) if act == "silu" else torch.sigmoid(z.double())
            want = plain.grouped_rms_norm(u * a if first else u, w.double(), parts, 1e-5) * (1.0 if first else a) * mult
            wide = torch.zeros(n, c + 8, dtype=dtype, device="cuda")
            ops.wide_norm_gate(o.cuda(), w.cuda(), 1e-5, wide[:, :c], parts, gate=z.cuda() if act else None, activation=act, gate_first=first,
                               skip=d.cuda() if skip else None, skip_x=x.cuda() if skip else None, mult=mult)  # fmt: skip
            assert torch.allclose(wide[:, :c].cpu().double(), want, atol=part_tol(dtype), rtol=part_tol(dtype)), (c, act, first)
            assert float(wide[:, c:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [1, 9, 40])
def test_summed_mixers(dtype, n):
    """Chunked attention and lightning attention in one input product and one output product, with their constants; then the
    following token on what they left."""
    from kvforge_b200.models.ritizen import ritizen_spec
    from kvforge_b200.config.ritizen_config import RitizenConfig
    from kvforge_b200.parts.base import build_part
    from ritizen_cases import layer, model, tensor_shapes

    for left, right, scales in ((attention(4, 2, 16, 24, chunk=7), lightning(2, 16, 8, [0.9, 0.99]), (0.6, -1.1)), (attention(3, 1, 12, 20, chunk=50), lightning(3, 10, 5, [0.5, 1.0, 0.97]), (0.0, 1.0))):
        rt = runtime(dtype)
        width, bs = 56, 4
        config = model(50, width, [layer("parallel", parallel(left, right, *scales), None)], eps=1e-5)
        part = build_part("mixer", ritizen_spec(RitizenConfig.from_dict(config)).layers[0].block.params["mixer"], "l0.mix.")
        shapes = {k[len("l0.mix.") :]: s for k, s in tensor_shapes(config).items() if k.startswith("l0.mix.")}
        w = rounded(shapes, dtype, 21)
        for branch in part.sub_parts():
            own = {k[len(branch.prefix) - len("l0.mix.") :]: v for k, v in w.items() if ("l0.mix." + k).startswith(branch.prefix)}
            bind(branch, own, dtype, rt)
        part.bind({}, rt)
        x = torch.randn(n + 1, width, generator=torch.Generator().manual_seed(2)).to(dtype)
        wd, xd = {"m." + k: v.double() for k, v in w.items()}, x.double()
        ref = scales[0] * plain.attention(xd, wd, "m.left.", left, 1e-5, *plain.keys_and_values(xd, wd, "m.left.", left, 1e-5))
        ref = ref + scales[1] * plain.lightning_attention(xd, wd, "m.right.", right, 1e-5)
        cache = pages(32, left["kv_heads"], bs, left["dim"], left["vdim"], dtype)
        cache.state = torch.zeros(2, *part.state_shape(), device="cuda")
        got = step_mixer(part, rt, x, bs, list(range(31, -1, -1)), [(0, n), (n, n + 1)], cache, slot=1)
        assert rel_rows(got, ref) < part_tol(dtype)
        assert float(cache.state[0].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps,c,act", [(4, 40, "silu"), (2, 33, None), (1, 16, "silu"), (6, 24, None)])
def test_convolution_with_a_bias(dtype, taps, c, act):
    """Short and long steps, whole and cut, against the plain convolution."""
    from kvforge_b200 import ops

    g = torch.Generator().manual_seed(4)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")  # noqa: E731
    t = 1100
    x, w, b = torch.randn(t, c, generator=g).to(dtype), torch.randn(c, taps, generator=g), torch.randn(c, generator=g)
    want = plain.causal_conv(x.double(), w.double(), b.double())
    want = plain.silu(want) if act else want
    for cuts in ([(0, t)], [(0, 1), (1, 4), (4, 6), (6, 30), (30, t)]):
        state = torch.zeros(3, (taps - 1) * c, device="cuda")
        out = torch.empty(t, c, dtype=dtype, device="cuda")
        for lo, hi in cuts:
            ops.causal_conv(x[lo:hi].cuda(), w.t().contiguous().cuda(), state, i32([0, hi - lo]), i32([1]), 1, out[lo:hi], activation=act, max_query_len=hi - lo, bias=b.cuda())
        assert torch.allclose(out.cpu().double(), want, atol=part_tol(dtype), rtol=part_tol(dtype)), cuts


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,width,ff", [(1, 64, 96), (7, 48, 50), (30, 64, 96), (200, 72, 640), (1100, 64, 4096)])
def test_plain_feed_forward_with_biases(dtype, n, width, ff):
    """For one token, a few and many, and an inner size that is no multiple of 8; its result joins the stream normed, with the bias
    of the second product inside the norm."""
    from kvforge_b200 import ops
    from kvforge_b200.parts.base import PartSpec, build_part

    rt = runtime(dtype, max_tokens=1200)
    part = build_part("ffn", PartSpec("plain_mlp", {"hidden_size": width, "intermediate_size": ff, "activation": "gelu_tanh", "bias": True}), "m.")
    w = rounded({"up": (ff, width), "up.b": (ff,), "down": (width, ff), "down.b": (width,)}, dtype, 6)
    bind(part, w, dtype, rt)
    g = torch.Generator().manual_seed(3)
    x, resid, weight = torch.randn(n, width, generator=g).to(dtype), torch.randn(n, width, generator=g), 1.0 + 0.2 * torch.randn(width, generator=g)
    ctx = context(rt, [n], [0], 4, [[0]], [0] * n)
    y = part.forward(ctx, x.cuda())
    assert isinstance(y, ops.Biased)
    r, out = resid.cuda(), torch.empty(n, width, dtype=dtype, device="cuda")
    ops.norm_step(r, ops.GatedWrite(y, post_w=weight.cuda()), None, out, 1e-5, centred=False)
    want = resid.double() + plain.rms_norm(plain.feed_forward(x.double(), {"m." + k: v.double() for k, v in w.items()}, "m."), weight.double(), 1e-5)
    assert rel_rows(r.cpu(), want) < part_tol(dtype)
    assert rel_rows(out.float().cpu(), want) < part_tol(dtype)


def test_positions_are_added_and_one_beyond_the_table_is_reported():
    from kvforge_b200.parts.base import PartSpec, build_part

    for dtype in (torch.float32, torch.bfloat16):
        rt = runtime(dtype)
        part = build_part("position", PartSpec("learned", {"rows": 20, "hidden_size": 37, "names": {"weight": "pos"}}), "")
        assert [part.tensor_name(k) for k in type(part).weight_decls(part.params)] == ["pos"]
        table = torch.randn(20, 37).to(dtype)
        part.bind({"weight": table.cuda()}, rt)
        resid = torch.randn(6, 37)
        ctx = context(rt, [4, 2], [16, 0], 4, [[0], [0]], [0] * 6)
        r = resid.cuda()
        part.embed(ctx, r)
        assert torch.allclose(r.cpu(), resid + table.float()[[16, 17, 18, 19, 0, 1]])
        rt.check_error_flag()
        ctx = context(rt, [2], [19], 4, [[0]], [0] * 2)
        r = resid[:2].cuda()
        part.embed(ctx, r)
        assert torch.allclose(r.cpu(), resid[:2] + torch.stack([table.float()[19], torch.zeros(37)]))
        with pytest.raises(RuntimeError, match="table of positions"):
            rt.check_error_flag()
