"""Small Ritizen configurations for the tests, weights made here (not by the package's random-weights mode), and
the plain implementation's logits for them.

The configurations differ from one another in every size and option: the order of the layers (each kind of mixer first,
last, twice in a row), layers that use an earlier layer's keys (right after it, far after it, two of one, of a chunked
layer), as many key heads as heads and a single key head, key and value sizes (equal and not, no multiple of 8), chunks
shorter than a page and longer than several, one group or several for B and C and for the norm, two to five taps and one,
state sizes that are and are not the value size, layers without a feed-forward, branch constants of one, negative and zero.
"""

from __future__ import annotations

import random

import torch

import plain_ritizen as plain
from mopilorn_cases import row_error, write_folder  # noqa: F401  (the folder writer and the error measure are the same)


def attention(heads, kv_heads, dim, vdim, scale=None, kv_from=None, chunk=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim**-0.5}
    if kv_from is not None:
        out["kv_from"] = kv_from
    if chunk is not None:
        out["mask"] = {"size": chunk}
    return out


def lightning(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def parallel(left, right, left_scale=0.7, right_scale=1.2):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def mamba2(heads, vdim, state, groups, conv=4, norm_groups=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(vocab, width, layers, eps=1e-6, max_positions=400):
    return {"architecture": "Ritizen", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps}, "layers": layers}


CASES: dict[str, dict] = {
    # the state space first; two layers over one layer's keys, one right after it and one last; a chunk shorter than a page
    "a": {
        "config": model(131, 64, [
            layer("mamba2", mamba2(4, 16, 24, 2, conv=3, norm_groups=2), 72),
            layer("attention", attention(4, 2, 16, 24), 40),
            layer("attention", attention(4, 2, 16, 24, kv_from=1), None),
            layer("parallel", parallel(attention(4, 2, 24, 16, chunk=11), lightning(2, 16, 24, [0.9, 0.99])), 64),
            layer("attention", attention(4, 2, 16, 24, kv_from=1, scale=0.4), 48),
        ], eps=1e-5),
        "block_size": 16,
    },
    # chunked attention first and last, with chunks of their own (cache groups of their own); a single key head; heads of
    # sizes that are no multiple of 8; an inner width and a feed-forward that are no multiple of 8; a long convolution
    "b": {
        "config": model(97, 48, [
            layer("parallel", parallel(attention(3, 1, 12, 20, chunk=37, scale=0.3), lightning(3, 10, 6, [0.5, 0.9375, 1.0]), 1.0, -0.6), 50),
            layer("mamba2", mamba2(3, 7, 5, 1, conv=5, norm_groups=3), None),
            layer("attention", attention(5, 5, 9, 13), 36),
            layer("mamba2", mamba2(6, 8, 16, 3, conv=2, norm_groups=1), 44),
            layer("parallel", parallel(attention(4, 4, 8, 8, chunk=5), lightning(1, 32, 8, [0.97]), -0.4, 1.0), None),
        ]),
        "block_size": 8,
    },
    # no state at all between two layers of attention, the second over the first one's keys; a width that is no multiple of 8;
    # pages of four tokens; one tap (no convolution state)
    "c": {
        "config": model(150, 44, [
            layer("attention", attention(6, 2, 16, 16), None),
            layer("attention", attention(6, 2, 16, 16, kv_from=0), 24),
            layer("mamba2", mamba2(2, 24, 40, 2, conv=1, norm_groups=4), 24),
            layer("mamba2", mamba2(2, 24, 40, 1, conv=4, norm_groups=1), 24),
        ], eps=1e-4),
        "block_size": 4,
    },
    # heads of 64 and of 128 (the tensor-core kernels in bfloat16), shared keys, a chunk of three pages, large states
    "d": {
        "config": model(211, 96, [
            layer("attention", attention(8, 2, 64, 64), 160),
            layer("parallel", parallel(attention(8, 4, 64, 64, chunk=48), lightning(2, 128, 64, [0.984375, 0.998])), 160),
            layer("attention", attention(8, 2, 64, 64, kv_from=0, scale=0.2), 96),
            layer("mamba2", mamba2(8, 32, 64, 2, norm_groups=2), None),
            layer("parallel", parallel(attention(4, 2, 128, 128, chunk=50), lightning(4, 64, 128, [0.9, 0.95, 0.99, 0.999]), 0.3, 0.9), 64),
        ], eps=1e-5),
        "block_size": 16,
    },
    # a layer over the keys of a chunked layer sees them all (its own mask decides), one over the same keys with the same chunk
    "e": {
        "config": model(88, 40, [
            layer("parallel", parallel(attention(4, 2, 16, 8, chunk=13), lightning(2, 8, 16, [0.8, 0.999]), 0.9, 0.5), 32),
            layer("attention", attention(4, 2, 16, 8, kv_from=0), 56),
            layer("mamba2", mamba2(1, 16, 8, 1, conv=3), 40),
            layer("parallel", parallel(attention(2, 1, 8, 16, chunk=21), lightning(1, 8, 8, [0.95]), 0.0, 1.0), 32),
            layer("attention", attention(4, 1, 8, 16, kv_from=3, chunk=21), 32),
        ]),
        "block_size": 4,
    },
}  # fmt: skip


def tensor_shapes(config: dict) -> dict[str, tuple[int, ...]]:
    """Checkpoint name -> shape, from the design's naming alone."""
    w = config["width"]
    out = {"embed": (config["vocab"], w), "pos": (config["max_positions"], w), "final.norm": (w,)}

    def attention_tensors(p, m, gate_rows, bias):
        h, g, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        rows = {"q": h * dk} if m.get("kv_from") is not None else {"q": h * dk, "k": g * dk, "v": g * dv}
        for name, n in rows.items():
            out[p + name] = (n, w)
            if bias:
                out[f"{p}{name}.b"] = (n,)
            if name != "v":
                out[f"{p}{name}.norm"] = (n,)
        out[p + "g"] = (gate_rows, w)
        out[p + "o"] = (w, h * dv)

    for i, ly in enumerate(config["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        out[p + "norm1"] = (w,)
        q = p + "mix."
        if ly["type"] == "attention":
            attention_tensors(q, m, m["heads"], False)
        elif ly["type"] == "parallel":
            left, r = m["left"], m["right"]
            attention_tensors(q + "left.", left, left["heads"] * left["vdim"], True)
            h, dk, dv = r["heads"], r["dim"], r["vdim"]
            q += "right."
            out.update({q + "q": (h * dk, w), q + "k": (h * dk, w), q + "v": (h * dv, w), q + "g": (h * dv, w), q + "o": (w, h * dv), q + "norm": (h * dv,)})
        else:
            h, inner, gn = m["heads"], m["heads"] * m["vdim"], m["groups"] * m["state"]
            out.update({q + "in": (2 * inner + 2 * gn + h, w), q + "conv": (inner + 2 * gn, m["conv"]), q + "conv.b": (inner + 2 * gn,), q + "dt_bias": (h,),
                        q + "A_log": (h,), q + "D": (h,), q + "norm": (inner,), q + "o": (w, inner)})  # fmt: skip
        if ly["mlp"]:
            ff = ly["mlp"]["ff"]
            out.update({p + "norm2": (w,), p + "mlp.up": (ff, w), p + "mlp.up.b": (ff,), p + "mlp.down": (w, ff), p + "mlp.down.b": (w,)})
    return out


def random_tensors(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Weights of order one where it matters, rounded to bfloat16 (what the files hold), as float32."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if name == "embed":
            t = r
        elif name == "pos":
            t = 0.5 * r
        elif leaf in ("norm1", "norm2", "norm", "D"):
            t = 1.0 + 0.2 * r
        elif leaf == "A_log":
            t = 0.7 * r - 1.0
        elif leaf == "dt_bias":
            t = 0.7 * r - 1.0
        elif leaf == "b":
            t = 0.2 * r
        elif leaf == "conv":
            t = 0.6 * r
        else:
            t = r * 1.5 / shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out


def plain_logits(config: dict, tensors: dict[str, torch.Tensor], tokens: list[int]) -> torch.Tensor:
    w = {k: v.double() for k, v in tensors.items()}
    return plain.logits(config, w, tokens)


def random_config(seed: int) -> dict:
    """A configuration drawn at random: widths that are and are not multiples of 8, one to twelve heads, one key head or several,
    head sizes from 4 to 128 that are and are not multiples of 8, chunks of 1 to 90 positions, one to six taps, one group or
    several, layers over earlier keys and layers without a feed-forward."""
    rng = random.Random(seed)
    width = rng.choice([8 * rng.randint(5, 18), 100, 52, 37])
    layers: list[dict] = []
    sources: list[int] = []
    for i in range(rng.randint(2, 6)):
        kind = rng.choice(["attention", "attention", "parallel", "mamba2"])
        size = lambda: rng.choice([4, 8, 12, 16, 24, 30, 40, 64, 128])  # noqa: E731
        if kind == "mamba2":
            groups = rng.choice([1, 1, 2, 3])
            heads, vdim = groups * rng.choice([1, 2, 4]), rng.choice([4, 8, 12, 16, 20, 32])
            ng = rng.choice([n for n in (1, 2, 4, 6) if (heads * vdim) % n == 0])
            mixer = mamba2(heads, vdim, rng.choice([4, 8, 13, 16, 32, 64, 100]), groups, conv=rng.randint(1, 6), norm_groups=ng)
        elif kind == "attention":
            if sources and rng.random() < 0.5:
                src = rng.choice(sources)
                m = layers[src]["mixer"]
                mixer = attention(m["kv_heads"] * rng.choice([1, 2, 3]), m["kv_heads"], m["dim"], m["vdim"], rng.uniform(0.1, 0.4), kv_from=src)
            else:
                g = rng.choice([1, 2, 3])
                mixer = attention(g * rng.choice([1, 2, 4]), g, size(), size(), rng.uniform(0.1, 0.4))
                sources.append(i)
        else:
            g = rng.choice([1, 2, 3])
            left = attention(g * rng.choice([1, 2, 3]), g, size(), size(), rng.uniform(0.1, 0.4), chunk=rng.randint(1, 90))
            heads = rng.choice([1, 2, 3, 6])
            right = lightning(heads, rng.choice([4, 8, 16, 20, 48]), rng.choice([4, 8, 12, 32, 40]), [rng.choice([0.5, 0.9, 0.99, 0.9995]) for _ in range(heads)])
            mixer = parallel(left, right, rng.uniform(0.2, 1.3), rng.uniform(-1.0, 1.3))
        layers.append(layer(kind, mixer, rng.choice([None, 8 * rng.randint(2, 12), 36, 50])))
    return model(rng.randint(30, 300), width, layers, eps=rng.choice([1e-5, 1e-6]), max_positions=rng.choice([256, 300]))
