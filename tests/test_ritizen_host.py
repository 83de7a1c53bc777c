"""What of the Ritizen decoder needs no GPU: the configuration and its names, the cache and state that the model asks
for, pages of chunks in the allocator, and the plain implementation's own pieces."""

from __future__ import annotations

import copy
import math
import random

import pytest
import torch

import plain_ritizen as plain
from ritizen_cases import CASES, random_config, random_tensors, tensor_shapes


def parsed(config):
    from kvforge_b200.config.registry import architecture_of
    from kvforge_b200.parts.model import DecoderModel

    arch = architecture_of(config)
    cfg = arch.parse_config(config)
    return arch, cfg, DecoderModel(arch.build_spec(cfg))


@pytest.mark.parametrize("name", sorted(CASES) + [f"drawn-{s}" for s in range(5, 12)])
def test_names_and_shapes_follow_the_configuration(name):
    config = CASES[name]["config"] if name in CASES else random_config(int(name.split("-")[1]))
    arch, cfg, model = parsed(config)
    got = {k: tuple(d.shape) for k, d in model.expected_weights().items() if not d.optional}
    assert got == tensor_shapes(config)
    again = arch.parse_config(cfg.to_hf_dict())  # what the file says comes back when it is written again
    assert again.layers == cfg.layers and again.max_position_embeddings == cfg.max_position_embeddings and again.eps == cfg.eps
    for ly, shape, owner in zip(config["layers"], model.state_shapes, model.call_group):
        m = ly["mixer"]
        if ly["type"] == "mamba2":
            channels = m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            assert shape == ((m["conv"] - 1) * channels + m["heads"] * m["state"] * m["vdim"],) and owner is None
        elif ly["type"] == "parallel":
            r = m["right"]
            assert shape == (r["heads"] * r["dim"] * r["vdim"],) and owner is not None
        else:
            assert shape is None and (owner is None) == (m.get("kv_from") is not None)


def test_cache_groups_of_shared_and_chunked_layers():
    groups = lambda model: sorted((g.need.kind, g.need.window or 0, g.calls) for g in model.groups)  # noqa: E731
    _, _, model = parsed(CASES["a"]["config"])
    assert groups(model) == [("chunk", 11, [3]), ("full", 0, [1])]
    _, _, model = parsed(CASES["b"]["config"])
    assert groups(model) == [("chunk", 5, [4]), ("chunk", 37, [0]), ("full", 0, [2])]
    assert [g.need.head_dim for g in model.groups] == [16, 16, 8] and [g.need.value_dim for g in model.groups] == [24, 16, 8]  # padded to 8
    # a chunked layer whose keys another layer sees beyond the chunk keeps them all; with the same chunk it gives them back
    _, _, model = parsed(CASES["e"]["config"])
    assert groups(model) == [("chunk", 21, [3]), ("full", 0, [0])]


def test_what_the_file_lacks_or_gets_wrong_is_named():
    from kvforge_b200.config.model_config import ConfigError
    from kvforge_b200.config.ritizen_config import RitizenConfig

    base = CASES["a"]["config"]
    for path, value in (
        (("layers", 0, "type"), "retention"),
        (("layers", 0, "mixer", "groups"), 3),
        (("layers", 0, "mixer", "norm_groups"), 5),
        (("layers", 0, "mixer", "conv"), 0),
        (("layers", 1, "mixer", "kv_heads"), 3),
        (("layers", 2, "mixer", "kv_from"), 0),  # a layer without keys
        (("layers", 2, "mixer", "kv_from"), 2),  # itself
        (("layers", 4, "mixer", "kv_from"), 2),  # a layer without keys of its own
        (("layers", 4, "mixer", "vdim"), 16),  # another shape than the source's
        (("layers", 3, "mixer", "right", "decay"), [0.9]),
        (("layers", 3, "mixer", "left", "mask", "size"), 0),
        (("layers", 3, "mixer", "left", "kv_from"), 1),
        (("layers", 0, "mlp", "kind"), "moe"),
    ):
        config = copy.deepcopy(base)
        d = config
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ConfigError):
            RitizenConfig.from_dict(config)
    for key in ("vocab", "width", "norm", "layers", "max_positions"):
        with pytest.raises(ConfigError):
            RitizenConfig.from_dict({k: v for k, v in base.items() if k != key})
    for key in ("left_scale", "right_scale", "left", "right"):
        config = copy.deepcopy(base)
        del config["layers"][3]["mixer"][key]
        with pytest.raises(ConfigError):
            RitizenConfig.from_dict(config)


def test_named_shapes():
    from kvforge_b200 import PRESETS

    for name in ("ritizen-tiny", "ritizen-1b", "ritizen-3b"):
        _, cfg, model = parsed(PRESETS[name].to_hf_dict())
        assert cfg.layers == PRESETS[name].layers
        assert {ly.type for ly in cfg.layers} == {"attention", "parallel", "mamba2"}
        assert any(c.kv_from is not None for c in model.spec.execution)


# ------------------------------------------------------------------ pages of chunks


def test_a_chunk_group_gives_back_the_pages_before_the_chunk():
    from kvforge_b200.cache.block_manager import BlockManager, GroupSpec

    bm = BlockManager(8, 4, groups=[GroupSpec("chunk", 10)])
    bm.allocate("a", 9, 9)
    assert [b >= 0 for b in bm.get_block_table("a")] == [True] * 3
    bm.append_slots("a", 10, 9)  # position 9 is the chunk's last: everything stays
    assert [b >= 0 for b in bm.get_block_table("a")] == [True] * 3
    bm.append_slots("a", 11, 10)  # position 10 begins a chunk: pages 0 and 1 hold positions 0 to 7 only, page 2 holds 8 to 11
    assert [b >= 0 for b in bm.get_block_table("a")] == [False, False, True]
    bm.append_slots("a", 25, 11)  # a portion that reaches over two borders: chunk 10 .. 19 is still seen by its first token
    assert [b >= 0 for b in bm.get_block_table("a")] == [False, False, True, True, True, True, True]
    bm.append_slots("a", 26, 25)
    assert [b >= 0 for b in bm.get_block_table("a")] == [False] * 5 + [True, True]
    bm.check_invariants()
    bm.free("a")
    assert bm.num_free_blocks == 8
    with pytest.raises(ValueError):
        GroupSpec("chunk")
    # a request longer than the pool fits when it is fed in portions
    assert bm.can_ever_fit(1000, 8) and not bm.can_ever_fit(1000, 40) and not BlockManager(8, 4).can_ever_fit(1000, 8)


@pytest.mark.parametrize("seed", range(4))
def test_chunk_groups_lose_no_page_under_random_orders(seed):
    from kvforge_b200.cache.block_manager import BlockManager, GroupSpec

    rng = random.Random(seed)
    bs, chunk = rng.choice([1, 4, 16]), rng.randint(1, 40)
    bm = BlockManager(64, bs, groups=[GroupSpec("full"), GroupSpec("chunk", chunk)])
    live: dict[str, int] = {}
    for k in range(300):
        if live and (rng.random() < 0.2 or len(live) > 3):
            rid = rng.choice(list(live))
            bm.free(rid)
            del live[rid]
        elif rng.random() < 0.3 and len(live) < 4:
            n = rng.randint(1, 20)
            if bm.can_allocate(n, n):
                bm.allocate(f"r{k}", n, n)
                live[f"r{k}"] = n
        elif live:
            rid = rng.choice(list(live))
            start, n = live[rid], rng.choice([1, 1, 2, 9, 30])
            if bm.can_append_slots(rid, start + n, start):
                bm.append_slots(rid, start + n, start)
                live[rid] = start + n
                for p in range(start, start + n):
                    for j in range(p - p % chunk, p + 1):  # every key a query of this step sees has a page
                        bm.slot(rid, j, 1)
                full, chunked = bm.get_block_table(rid, 0), bm.get_block_table(rid, 1)
                assert len(full) == len(chunked) and all(b >= 0 for b in full)
                first = (start - start % chunk) // bs
                assert all(b < 0 for b in chunked[:first])
        bm.check_invariants()


# ------------------------------------------------------------------ the plain implementation's own pieces


def test_plain_pieces():
    # a chunk's positions see one another's past and nothing else
    m = plain.chunked_causal(7, 3)
    assert [row.nonzero().flatten().tolist() for row in m] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]
    # parts of a row have root mean squares of their own
    y = torch.tensor([[3.0, -3.0, 1.0, 1.0]], dtype=torch.float64)
    w = torch.tensor([1.0, 2.0, 3.0, 4.0], dtype=torch.float64)
    assert torch.allclose(plain.grouped_rms_norm(y, w, 2, 0.0), torch.tensor([[1.0, -2.0, 3.0, 4.0]], dtype=torch.float64))
    assert torch.allclose(plain.grouped_rms_norm(y, w, 1, 0.0), y / 5.0**0.5 * w)
    # the convolution: the last tap is the token's own
    x = torch.tensor([[1.0], [2.0], [3.0]], dtype=torch.float64)
    taps, bias = torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64), torch.tensor([0.5], dtype=torch.float64)
    assert plain.causal_conv(x, taps, bias).flatten().tolist() == [1.5, 12.5, 123.5]
    z = torch.tensor([-40.0, -1.0, 0.0, 3.0, 60.0], dtype=torch.float64)
    assert torch.allclose(plain.softplus(z), torch.tensor([math.log1p(math.exp(v)) if v < 50 else v for v in z.tolist()], dtype=torch.float64))


def test_plain_recurrences_are_decaying_sums():
    """The walks against their sums written out: ``o_t = sum_(s <= t) a^(t-s) (q_t . k_s) v_s``, and for the state space the
    product of the decays between the two tokens."""
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    q, k, v = r(7, 2, 4), r(7, 2, 4), r(7, 2, 3)
    o = plain.fixed_decay_walk(q, k, v, [0.8, 1.0])
    for h, a in enumerate((0.8, 1.0)):
        want = torch.stack([sum(a ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1)) for t in range(7)])
        assert torch.allclose(o[:, h], want)
    x, b, c, dt, a_log, skip = r(6, 4, 3), r(6, 2, 5), r(6, 2, 5), r(6, 4).abs(), r(4), r(4)
    y = plain.state_space_walk(x, b, c, dt, a_log, skip)
    for h in range(4):
        grp, rate = h // 2, math.exp(float(a_log[h]))
        for t in range(6):
            want = skip[h] * x[t, h]
            for s in range(t + 1):
                want = want + math.exp(-rate * float(dt[s + 1 : t + 1, h].sum())) * float(dt[s, h]) * (c[t, grp] @ b[s, grp]) * x[s, h]
            assert torch.allclose(y[t, h], want)


def test_plain_model_sees_its_chunk_and_carries_its_states():
    """A change of a token shows in a later position's logits inside the chunk only, when attention is all there is, and at any
    distance once a recurrence or an uncut layer carries it."""
    left = {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 0.35, "mask": {"size": 6}}
    right = {"heads": 1, "dim": 4, "vdim": 4, "decay": [0.9]}
    config = {"architecture": "Ritizen", "vocab": 50, "width": 32, "max_positions": 40, "norm": {"eps": 1e-5},
              "layers": [{"type": "parallel", "mlp": None, "mixer": {"left": left, "right": right, "left_scale": 1.0, "right_scale": 0.0}}]}  # fmt: skip
    w = {k: v.double() for k, v in random_tensors(config, 3).items()}
    base = list(range(10, 30))

    def moved(j):
        toks = list(base)
        toks[j] += 1
        return float((plain.logits(config, w, toks)[16] - plain.logits(config, w, base)[16]).abs().max()) > 1e-9

    assert [j for j in range(17) if moved(j)] == [12, 13, 14, 15, 16]
    config["layers"][0]["mixer"]["right_scale"] = 0.5
    assert all(moved(j) for j in range(17))
