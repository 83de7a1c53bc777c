"""Small Latuzen configurations for the tests, weights made here (not by the package's random-weights mode), and
the plain implementation's logits for them.

The configurations differ from one another in every size and option: the order of the layers (each kind of mixer first and
last), layers that use an earlier layer's keys (right after it, far after it, two of one, with windows shorter and longer
than the source's), as many key heads as heads and a single key head, key and value sizes (equal and not, no multiple
of 8), windows shorter than a page and longer than several, rotations of a whole head and of a part of it, with and
without scaling (and with ramps that begin below zero, end past the last pair, or have no width), memories of one head and of several with key sizes
below and above the value size, small and large caps, groups of one member and one group, no identity experts and more of them than experts, one
expert a token and several, layers without a feed-forward.
"""

from __future__ import annotations

import random

import torch

import plain_latuzen as plain
from mopilorn_cases import row_error, write_folder  # noqa: F401  (the folder writer and the error measure are the same)


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def rotation(dims, base, scaling=None):
    return {"dims": dims, "base": base, **({"scaling": scaling} if scaling else {})}


def attention(heads, kv_heads, dim, vdim, window, rot, scale=None, kv_from=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim**-0.5, "mask": {"size": window}, "rot": rot}
    if kv_from is not None:
        out["kv_from"] = kv_from
    return out


def memory(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, identity, top, groups, keep, scale):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}}


def own(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def both(left, right, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def model(vocab, width, layers, eps=1e-6):
    return {"architecture": "Latuzen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


PART = rotation(8, 1000.0, yarn(4.0, 64, 8.0, 1.0))
WHOLE = rotation(16, 5000.0, yarn(3.0, 40, 6.0, 0.5))

CASES: dict[str, dict] = {
    # a window shorter than a page and readers with a shorter and a longer one; the memory in the middle; one member a group
    "a": {
        "config": model(131, 64, [
            own(attention(4, 2, 16, 24, 11, PART), dense(72)),
            own(attention(6, 2, 16, 24, 30, PART, scale=0.4, kv_from=0), moe(40, 5, 1, 2, 6, 3, 1.7)),
            both(attention(4, 2, 24, 16, 19, rotation(24, 700.0)), memory(2, 16, 24, 15.0), dense(64)),
            own(attention(2, 2, 16, 24, 5, PART, kv_from=0), None),
        ], eps=1e-5),
        "block_size": 16,
    },
    # the memory first and last; a single key head; heads of sizes that are no multiple of 8; inner sizes and a width that are no multiple
    # of 8; more identity experts than experts; one expert a token; one group
    "b": {
        "config": model(97, 44, [
            both(attention(3, 1, 12, 20, 37, rotation(6, 100.0), scale=0.3), memory(3, 10, 6, 2.5), moe(50, 3, 5, 1, 2, 1, 2.5)),
            own(attention(5, 5, 10, 14, 23, rotation(10, 300.0, yarn(2.0, 500, 32.0, 1.0))), dense(36)),
            own(attention(5, 5, 10, 14, 23, rotation(10, 300.0, yarn(2.0, 500, 32.0, 1.0)), kv_from=1), moe(24, 4, 0, 3, 1, 1, 0.6)),
            both(attention(4, 4, 8, 9, 5, rotation(8, 50.0)), memory(1, 32, 7, 0.8), None),
        ]),
        "block_size": 8,
    },
    # pages of four tokens, a window of one key, no identity experts and one, a ramp without width (the frequencies switch at one pair)
    "c": {
        "config": model(150, 40, [
            own(attention(6, 2, 16, 16, 1, WHOLE), None),
            both(attention(2, 2, 16, 16, 64, rotation(2, 10.0)), memory(4, 20, 8, 30.0), moe(16, 8, 0, 4, 4, 2, 3.0)),
            own(attention(6, 3, 16, 8, 50, rotation(16, 20000.0, yarn(16.0, 7, 1.0, 1.0))), moe(24, 7, 1, 2, 2, 2, 1.0)),
            own(attention(3, 3, 16, 8, 45, rotation(16, 20000.0, yarn(16.0, 7, 1.0, 1.0)), kv_from=2), dense(24)),
        ], eps=1e-4),
        "block_size": 4,
    },
    # heads of 64 and of 128 (the tensor-core kernels in bfloat16), inner sizes over which the decode products run in slices, large memories
    "d": {
        "config": model(211, 96, [
            own(attention(8, 2, 64, 64, 48, rotation(64, 10000.0, yarn(2.0, 128, 16.0, 1.0))), dense(1024)),
            own(attention(16, 2, 64, 64, 90, rotation(64, 10000.0, yarn(2.0, 128, 16.0, 1.0)), scale=0.2, kv_from=0), dense(640)),
            both(attention(8, 4, 64, 64, 70, rotation(32, 500.0)), memory(2, 128, 64, 12.0), moe(160, 6, 2, 3, 2, 1, 1.3)),
            own(attention(4, 2, 128, 128, 33, rotation(96, 10000.0)), moe(64, 12, 4, 2, 4, 2, 2.0)),
            both(attention(4, 2, 128, 128, 100, rotation(128, 10000.0)), memory(4, 64, 128, 6.0), dense(512)),
        ], eps=1e-5),
        "block_size": 16,
    },
}  # fmt: skip


def tensor_shapes(config: dict) -> dict[str, tuple[int, ...]]:
    """Checkpoint name -> shape, from the design's naming alone."""
    w = config["width"]
    out = {"embed": (config["vocab"], w), "head": (config["vocab"], w), "final.norm": (w,), "final.norm.b": (w,)}
    for i, ly in enumerate(config["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        out[p + "norm1"] = out[p + "norm1.b"] = (w,)
        q = p + "mix."
        if ly["type"] == "attention":
            h, g, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            rows = {"q": h * dk} if m.get("kv_from") is not None else {"q": h * dk, "k": g * dk, "v": g * dv}
            for name, n in rows.items():
                out[q + name], out[f"{q}{name}.b"] = (n, w), (n,)
                if name != "v":
                    out[f"{q}{name}.norm"] = (n,)
            out[q + "o"] = (w, h * dv)
        else:
            left, r = m["left"], m["right"]
            h, g, dk, dv = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
            s = q + "left."
            out.update({s + "q": (h * dk, w), s + "k": (g * dk, w), s + "v": (g * dv, w), s + "q.norm": (dk,), s + "k.norm": (dk,), s + "o": (w, h * dv)})
            h, dk, dv = r["heads"], r["dim"], r["vdim"]
            s = q + "right."
            out.update({s + "q": (h * dk, w), s + "k": (h * dk, w), s + "v": (h * dv, w), s + "g": (h * dv, w), s + "o": (w, h * dv), s + "norm": (h * dv,),
                        s + "i": (h, w), s + "i.b": (h,), s + "f": (h, w), s + "f.b": (h,), q + "left.out": (w,), q + "right.out": (w,)})  # fmt: skip
        f = p + "mlp."
        mlp = ly["mlp"]
        if mlp and mlp["kind"] == "dense":
            out.update({f + "gate": (mlp["ff"], w), f + "up": (mlp["ff"], w), f + "down": (w, mlp["ff"])})
        elif mlp:
            ff, r = mlp["expert"]["ff"], mlp["router"]
            n = r["experts"] + r.get("identity", 0)
            out.update({f + "router": (n, w), f + "correction": (n,)})
            for e in range(r["experts"]):
                out.update({f"{f}e{e}.gate": (ff, w), f"{f}e{e}.up": (ff, w), f"{f}e{e}.down": (w, ff)})
    return out


def random_tensors(config: dict, seed: int, fixed_choice: bool = False) -> dict[str, torch.Tensor]:
    """Weights of order one where it matters, rounded to bfloat16 (what the files hold), as float32.  The heads of a memory forget
    at different rates, some hardly at all.  ``fixed_choice``: the corrections lie so far apart that they alone decide which
    experts a token uses (rounding cannot move a token to other experts than the plain model's)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if name == "embed":
            t = r
        elif leaf in ("norm1", "norm", "out"):
            t = 1.0 + 0.2 * r
        elif name.endswith(".f.b"):
            t = 2.0 + 2.0 * r
        elif leaf == "b":
            t = 0.3 * r
        elif leaf == "correction":
            t = 1.5 * torch.randperm(shape[0], generator=g).float() - shape[0] if fixed_choice else 0.1 * r
        elif leaf == "router":
            t = r * 2.0 / shape[-1] ** 0.5
        else:
            t = r * 1.5 / shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out


def plain_logits(config: dict, tensors: dict[str, torch.Tensor], tokens: list[int]) -> torch.Tensor:
    w = {k: v.double() for k, v in tensors.items()}
    return plain.logits(config, w, tokens)


def random_config(seed: int) -> dict:
    """A configuration drawn at random: widths that are and are not multiples of 8, one to twelve heads, one key head or several,
    head sizes from 4 to 128, windows of 1 to 90 positions, any part of a head turning, every grouping of up to twelve
    experts and up to six identity experts, layers over earlier keys and layers without a feed-forward."""
    rng = random.Random(seed)
    width = rng.choice([8 * rng.randint(5, 18), 100, 52, 37])
    layers: list[dict] = []
    sources: list[int] = []

    def rot(dim, scaled):
        s = yarn(rng.choice([1.0, 2.0, 5.0, 32.0]), rng.choice([16, 100, 2048]), rng.choice([1.0, 8.0, 32.0]), rng.choice([0.5, 1.0])) if scaled else None
        return rotation(2 * rng.randint(1, dim // 2), rng.choice([50.0, 10000.0, 1e6]), s)

    def ffn():
        kind = rng.choice(["none", "dense", "moe", "moe"])
        if kind == "none":
            return None
        if kind == "dense":
            return dense(rng.choice([8 * rng.randint(2, 40), 36, 50]))
        groups = rng.choice([1, 2, 3, 4])
        n = groups * rng.randint(1, 4)
        identity = rng.randint(0, min(6, n - 1))
        keep = rng.randint(1, groups)
        return moe(rng.choice([16, 24, 30, 40]), n - identity, identity, rng.randint(1, min(4, keep * (n // groups))), groups, keep, rng.choice([0.7, 1.0, 2.5]))

    for i in range(rng.randint(2, 6)):
        size = lambda: rng.choice([4, 8, 12, 16, 24, 30, 40, 64, 128])  # noqa: E731
        if rng.random() < 0.6:
            if sources and rng.random() < 0.5:
                src = rng.choice(sources)
                m = layers[src]["mixer"]
                mixer = attention(m["kv_heads"] * rng.choice([1, 2, 3]), m["kv_heads"], m["dim"], m["vdim"], rng.randint(1, 90), m["rot"], rng.uniform(0.1, 0.4), kv_from=src)
            else:
                g, dim = rng.choice([1, 2, 3]), size()
                mixer = attention(g * rng.choice([1, 2, 4]), g, dim, size(), rng.randint(1, 90), rot(dim, rng.random() < 0.8), rng.uniform(0.1, 0.4))
                sources.append(i)
            layers.append(own(mixer, ffn()))
        else:
            g, dim = rng.choice([1, 2, 3]), size()
            left = attention(g * rng.choice([1, 2, 3]), g, dim, size(), rng.randint(1, 90), rot(dim, False), rng.uniform(0.1, 0.4))
            layers.append(both(left, memory(rng.choice([1, 2, 3, 6]), rng.choice([4, 8, 16, 20, 48]), rng.choice([4, 8, 12, 31, 40]), rng.choice([0.5, 4.0, 15.0])), ffn()))
    return model(rng.randint(30, 300), width, layers, eps=rng.choice([1e-5, 1e-6]))
