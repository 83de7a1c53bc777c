"""What of the Latuzen decoder needs no GPU: the configuration and its names, the cache and state that the model asks for, the scaled
frequencies, and the plain implementation's own pieces."""

from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_latuzen as plain
from latuzen_cases import CASES, attention, both, dense, memory, model, own, random_config, random_tensors, rotation, tensor_shapes, yarn


def parsed(config):
    from kvforge_b200.config.registry import architecture_of
    from kvforge_b200.parts.model import DecoderModel

    arch = architecture_of(config)
    cfg = arch.parse_config(config)
    return arch, cfg, DecoderModel(arch.build_spec(cfg))


@pytest.mark.parametrize("name", sorted(CASES) + [f"drawn-{s}" for s in range(5, 15)])
def test_names_and_shapes_follow_the_configuration(name):
    config = CASES[name]["config"] if name in CASES else random_config(int(name.split("-")[1]))
    arch, cfg, m = parsed(config)
    got = {k: tuple(d.shape) for k, d in m.expected_weights().items()}
    assert got == tensor_shapes(config)
    again = arch.parse_config(cfg.to_hf_dict())  # what the file says comes back when it is written again
    assert again.layers == cfg.layers and again.eps == cfg.eps and (again.vocab_size, again.hidden_size) == (cfg.vocab_size, cfg.hidden_size)
    for ly, shape, owner in zip(config["layers"], m.state_shapes, m.call_group):
        if ly["type"] == "parallel":
            r = ly["mixer"]["right"]
            columns = r["vdim"] + 1
            floats = r["heads"] * (r["dim"] * (columns + -columns % 4) + 1)  # the matrix, the key sum, the running maximum
            assert shape == (floats + -floats % 4,) and owner is not None
        else:
            assert shape is None and (owner is None) == (ly["mixer"].get("kv_from") is not None)


def test_a_cache_keeps_what_its_longest_reader_sees():
    groups = lambda m: sorted((g.need.kind, g.need.window or 0, g.calls) for g in m.groups)  # noqa: E731
    _, _, m = parsed(CASES["a"]["config"])
    assert groups(m) == [("window", 19, [2]), ("window", 30, [0])]
    assert [m.blocks[i].mixer_part().window for i in (0, 1, 3)] == [11, 30, 5]
    _, _, m = parsed(CASES["b"]["config"])
    assert groups(m) == [("window", 5, [3]), ("window", 23, [1]), ("window", 37, [0])]
    assert sorted((g.need.head_dim, g.need.value_dim) for g in m.groups) == [(8, 16), (16, 16), (16, 24)]  # padded to 8
    config = copy.deepcopy(CASES["a"]["config"])
    del config["layers"][3]["mixer"]["mask"]  # a reader that sees everything
    _, _, m = parsed(config)
    assert groups(m) == [("full", 0, [0]), ("window", 19, [2])]


def test_what_the_file_lacks_or_gets_wrong_is_named():
    from kvforge_b200.config.latuzen_config import LatuzenConfig
    from kvforge_b200.config.model_config import ConfigError

    base = CASES["a"]["config"]
    for path, value in (
        (("layers", 0, "type"), "mamba2"),
        (("layers", 0, "mixer", "kv_heads"), 3),
        (("layers", 0, "mixer", "rot", "dims"), 7),
        (("layers", 0, "mixer", "rot", "dims"), 18),
        (("layers", 0, "mixer", "rot", "scaling", "factor"), 0),
        (("layers", 0, "mixer", "mask", "size"), 0),
        (("layers", 1, "mixer", "kv_from"), 1),  # itself
        (("layers", 1, "mixer", "kv_from"), 2),  # a later layer
        (("layers", 3, "mixer", "kv_from"), 1),  # a layer without keys of its own
        (("layers", 3, "mixer", "kv_from"), 2),  # a layer of the other kind
        (("layers", 1, "mixer", "vdim"), 16),  # another shape than the source's
        (("layers", 1, "mlp", "router", "groups", "count"), 4),
        (("layers", 1, "mlp", "router", "groups", "keep"), 7),
        (("layers", 1, "mlp", "router", "top"), 4),  # more than the kept groups hold
        (("layers", 1, "mlp", "router", "experts"), 0),
        (("layers", 2, "mixer", "right", "gate_cap"), 0.0),
        (("layers", 2, "mixer", "left", "kv_from"), 0),
        (("layers", 0, "mlp", "kind"), "plain"),
    ):
        config = copy.deepcopy(base)
        d = config
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ConfigError):
            LatuzenConfig.from_dict(config)
    for key in ("vocab", "width", "norm", "layers"):
        with pytest.raises(ConfigError):
            LatuzenConfig.from_dict({k: v for k, v in base.items() if k != key})
    for at in (("mixer", "left"), ("mixer", "right"), ("mixer", "right", "gate_cap"), ("mixer", "left", "scale"), ("mlp", "ff")):
        config = copy.deepcopy(base)
        d = config["layers"][2]
        for k in at[:-1]:
            d = d[k]
        del d[at[-1]]
        with pytest.raises(ConfigError):
            LatuzenConfig.from_dict(config)


def test_named_shapes():
    from kvforge_b200 import PRESETS

    for name in ("latuzen-tiny", "latuzen-1b", "latuzen-3b"):
        _, cfg, m = parsed(PRESETS[name].to_hf_dict())
        assert cfg.layers == PRESETS[name].layers
        assert {ly.type for ly in cfg.layers} == {"attention", "parallel"}
        assert any(c.kv_from is not None for c in m.spec.execution)


# ------------------------------------------------------------------ scaled frequencies


def test_scaled_frequencies_against_values_by_hand():
    """Sixteen dims, base 10,000, original context 100: the pair that turns once lies at 16 ln(100 / 2 pi) / (2 ln 10000) = 2.404, the one
    that turns eight times at 0.598; so pair 0 keeps its frequency, pairs 3 to 7 are divided by the factor, and pairs 1 and 2 lie a third
    and two thirds between."""
    from kvforge_b200.parts.rope import yarn_scale

    f = [10000.0 ** (-i / 8) for i in range(8)]
    want = [f[0], f[1] * (2 / 3 + 1 / 12), f[2] * (1 / 3 + 2 / 12), *(v / 4 for v in f[3:])]
    assert torch.allclose(yarn_scale(16, 10000.0, 4.0, 100.0, 8.0, 1.0).double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6)
    assert plain.frequencies(rotation(16, 10000.0, yarn(4.0, 100, 8.0, 1.0))) == pytest.approx(want, rel=1e-12)
    # ramps that begin below zero (clamped), that end past the last pair (clamped to dims - 1 = 15, not to the last pair), that have no width
    for dims, base, s, ramp in ((16, 10000.0, yarn(4.0, 10, 8.0, 1.0), [0, 1, 1, 1, 1, 1, 1, 1]), (8, 10.0, yarn(4.0, 5000, 8.0, 1.0), [0, 0, 0, 0]),
                                (8, 40.0, yarn(4.0, 5000, 800.0, 1.0), [0, 1 / 7, 2 / 7, 3 / 7]), (8, 10.0, yarn(4.0, 1, 1.0, 1.0), [0, 1, 1, 1])):  # fmt: skip
        want = [base ** (-2 * i / dims) * (r / 4 + 1 - r) for i, r in enumerate(ramp)]
        assert plain.frequencies(rotation(dims, base, s)) == pytest.approx(want, rel=1e-12), (dims, base, s)
        got = yarn_scale(dims, base, s["factor"], s["original"], s["fast"], s["slow"]).double()
        assert torch.allclose(got, torch.tensor(want, dtype=torch.float64), rtol=1e-6), (dims, base, s)


def test_the_rotation_carries_the_size_of_its_pairs():
    from kvforge_b200.parts.base import PartSpec, build_part

    part = build_part("position", PartSpec("rotary", {"head_dim": 16, "theta": 1e4, "scaling": {"type": "yarn", **yarn(4.0, 100, 8.0, 1.0)}}))
    assert part.magnitude == pytest.approx(0.1 * math.log(4.0) + 1.0)
    assert torch.equal(part.inv_freq_host().double(), torch.tensor(plain.frequencies(rotation(16, 1e4, yarn(4.0, 100, 8.0, 1.0)))).float().double())
    assert build_part("position", PartSpec("rotary", {"head_dim": 16, "theta": 1e4})).magnitude == 1.0
    with pytest.raises(ValueError):
        build_part("position", PartSpec("rotary", {"head_dim": 16, "theta": 1e4, "scaling": {"type": "yarn", **yarn(0.0, 100, 8.0, 1.0)}}))


# ------------------------------------------------------------------ the plain implementation's own pieces


def test_plain_pieces():
    m = plain.window_mask(5, 2)
    assert [row.nonzero().flatten().tolist() for row in m] == [[0], [0, 1], [1, 2], [2, 3], [3, 4]]
    x = torch.tensor([[1.0, 2.0, 6.0, 3.0]], dtype=torch.float64)  # mean 3, mean squared deviation 3.5
    w, b = torch.tensor([1.0, 2.0, 1.0, 1.0], dtype=torch.float64), torch.tensor([0.0, 0.0, 1.0, 5.0], dtype=torch.float64)
    r = 4.0**-0.5
    assert torch.allclose(plain.layer_norm(x, w, b, 0.5), torch.tensor([[-2 * r, -2 * r, 3 * r + 1, 5.0]], dtype=torch.float64))
    z = torch.tensor([-40.0, -1.0, 0.0, 3.0, 60.0], dtype=torch.float64)
    assert torch.allclose(plain.log_sigmoid(z), torch.nn.functional.logsigmoid(z))
    # one key whose score equals the sink's takes half the weight; far larger, all of it; far smaller, none
    q, v = torch.ones(1, 1, 2, dtype=torch.float64), torch.ones(1, 1, 1, dtype=torch.float64)
    see = plain.window_mask(1, 1)
    for score, part in ((0.0, 0.5), (30.0, 1.0), (-30.0, 0.0)):
        k = torch.full((1, 1, 2), score / 2, dtype=torch.float64)
        assert float(plain.attend(q, k, v, 1.0, see, True)) == pytest.approx(part, abs=1e-9)
        assert float(plain.attend(q, k, v, 1.0, see, False)) == pytest.approx(1.0)
    # pairs: neighbours, or the two halves of what turns; the rest passes
    x = torch.arange(1.0, 7.0, dtype=torch.float64).reshape(1, 1, 6).repeat(2, 1, 1)
    rot = rotation(4, 100.0)
    a0, a1 = 1.0, 0.1
    rows = [plain.rotate(x, rot, inter)[1, 0].tolist() for inter in (True, False)]
    turn = lambda u, v, a: (u * math.cos(a) - v * math.sin(a), v * math.cos(a) + u * math.sin(a))  # noqa: E731
    (p0, p1), (p2, p3) = turn(1, 2, a0), turn(3, 4, a1)
    assert rows[0] == pytest.approx([p0, p1, p2, p3, 5, 6])
    (s0, s2), (s1, s3) = turn(1, 3, a0), turn(2, 4, a1)
    assert rows[1] == pytest.approx([s0, s1, s2, s3, 5, 6])


def test_plain_router_ranks_groups_by_their_best_member():
    """Scores follow the softmax, the choice the corrected scores (which may be negative), groups their largest member; the weights are
    the scores alone, scaled."""
    logits = torch.tensor([[1.0, 0.0, 2.0, -1.0, 0.5, 0.4]], dtype=torch.float64)
    w = {"router": torch.eye(6, dtype=torch.float64), "correction": torch.tensor([-9.0, -9.0, -9.0, -2.0, -3.0, -2.5], dtype=torch.float64)}
    r = {"experts": 4, "identity": 2, "top": 1, "groups": {"count": 3, "keep": 1}, "scale": 2.0}
    ids, weights = plain.route(logits, w, "", r)
    s = torch.softmax(logits[0], 0)
    assert ids == [[3]] and float(weights[0, 0]) == pytest.approx(2 * float(s[3]))  # the middle group: -9 beside -2 + s beats -3 beside -2.5
    ids, weights = plain.route(logits, w, "", {**r, "top": 2, "groups": {"count": 3, "keep": 2}})
    assert ids == [[3, 5]] and float(weights[0, 1]) == pytest.approx(2 * float(s[5]))
    # an identity expert hands its input on
    w.update({f"e{e}.{n}": torch.zeros(6, 6, dtype=torch.float64) for e in range(4) for n in ("gate", "up", "down")})
    out = plain.routed_experts(logits, w, "", {"router": {**r, "top": 2, "groups": {"count": 3, "keep": 2}}})
    assert torch.allclose(out, 2 * s[5] * logits)


def test_plain_memory_is_a_normalized_decaying_sum():
    """The walk against its sums written out without a running maximum: with ``A = log of a token's weight at t``,
    ``o_t = sum e^A (q . k) v / max(|sum e^A (q . k)|, 1)`` (the state starts relative to e^0), up to the 1e-6 beside the divisor."""
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    t, h = 8, 2
    q, k, v = r(t, h, 4), r(t, h, 4), r(t, h, 3)
    log_in, log_keep = 2.0 * r(t, h), plain.log_sigmoid(2.0 * r(t, h))
    o = plain.matrix_memory_walk(q, k, v, log_in, log_keep)
    top = torch.zeros(h, dtype=torch.float64)
    for s in range(t):
        top = torch.maximum(log_keep[s] + top, log_in[s])
        for head in range(h):
            weight = [math.exp(float(log_in[j, head] + log_keep[j + 1 : s + 1, head].sum())) * float(q[s, head] @ k[j, head]) for j in range(s + 1)]
            num = sum(a * v[j, head] for j, a in enumerate(weight))
            want = num / (max(abs(sum(weight)), 1.0) + 1e-6 * math.exp(float(top[head])))
            assert torch.allclose(o[s, head], want, rtol=1e-9), (s, head)


def test_plain_model_sees_its_window_and_carries_its_memory():
    """A change of a token shows in a later position's logits inside the window only, when attention is all there is, and at any
    distance once a memory carries it."""
    att = attention(2, 1, 8, 8, 6, rotation(8, 100.0))
    base = list(range(10, 30))

    def moved(config, j):
        w = {k: v.double() for k, v in random_tensors(config, 3).items()}
        toks = list(base)
        toks[j] += 1
        return float((plain.logits(config, w, toks)[16] - plain.logits(config, w, base)[16]).abs().max()) > 1e-12

    config = model(50, 32, [own(att, dense(16))])
    assert [j for j in range(17) if moved(config, j)] == [11, 12, 13, 14, 15, 16]
    config = model(50, 32, [both(att, memory(1, 4, 4, 5.0), None)])
    assert all(moved(config, j) for j in range(17))
