"""Typed configuration of the Latuzen decoder, read from its ``config.json``.

The file gives every size and every constant that differs between models of the design::

    {"architecture": "Latuzen", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "attention" | "parallel", "mixer": {...}, "mlp": {...} | null}, ...]}

An ``attention`` mixer: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (the window), ``rot`` (``dims``, ``base`` and, where the
frequencies are scaled, ``scaling``: ``factor``, ``original``, ``fast``, ``slow``) and, in a layer that uses an earlier layer's keys and values,
``kv_from``.  A ``parallel`` mixer: ``left`` (the same, without ``kv_from``) and ``right`` (``heads``, ``dim``, ``vdim``, ``gate_cap``).  A
feed-forward: ``kind`` ``dense`` with ``ff``, or ``moe`` with ``expert.ff`` and ``router`` (``experts``, ``identity``, ``top``, ``groups.count``,
``groups.keep``, ``scale``).  Nothing here has a default that stands for a size; a part of the file that may be absent (a mask, a
scaling, groups, identity experts) stands for the mechanism's absence.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from .model_config import ConfigError

ARCHITECTURE = "Latuzen"


def _need(d, key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        raise ConfigError(f"config.json lacks {where}{key}")
    return d[key]


def _positive(d, key: str, where: str) -> int:
    v = int(_need(d, key, where))
    if v <= 0:
        raise ConfigError(f"{where}{key} must be positive")
    return v


@dataclass(frozen=True)
class YarnConfig:
    factor: float
    original: float
    fast: float
    slow: float

    @classmethod
    def from_dict(cls, d: dict, where: str) -> YarnConfig:
        out = cls(**{k: float(_need(d, k, where)) for k in ("factor", "original", "fast", "slow")})
        if min(out.factor, out.original, out.fast, out.slow) <= 0:
            raise ConfigError(f"{where}factor, original, fast and slow must be positive")
        return out

    def to_dict(self) -> dict:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class RotationConfig:
    dims: int
    base: float
    scaling: YarnConfig | None = None

    @classmethod
    def from_dict(cls, d: dict, where: str, head: int) -> RotationConfig:
        dims = int(_need(d, "dims", where))
        if dims <= 0 or dims % 2 or dims > head:
            raise ConfigError(f"{where}dims must be even, positive and at most the head's size")
        base = float(_need(d, "base", where))
        if base <= 1:
            raise ConfigError(f"{where}base must be above one")
        s = d.get("scaling")
        return cls(dims, base, YarnConfig.from_dict(s, where + "scaling.") if s else None)

    def to_dict(self) -> dict:
        return {"dims": self.dims, "base": self.base, **({"scaling": self.scaling.to_dict()} if self.scaling else {})}


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None = None
    rot: RotationConfig | None = None
    kv_from: int | None = None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> AttentionConfig:
        sizes = {k: _positive(d, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
        mask, rot, source = d.get("mask"), d.get("rot"), d.get("kv_from")
        out = cls(
            **sizes, scale=float(_need(d, "scale", where)), window=_positive(mask, "size", where + "mask.") if mask else None,
            rot=RotationConfig.from_dict(rot, where + "rot.", sizes["dim"]) if rot else None, kv_from=int(source) if source is not None else None,
        )  # fmt: skip
        if out.heads % out.kv_heads:
            raise ConfigError(f"{where}heads must be a multiple of kv_heads")
        return out

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.window is not None:
            out["mask"] = {"size": self.window}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class MemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, d: dict, where: str) -> MemoryConfig:
        out = cls(**{k: _positive(d, k, where) for k in ("heads", "dim", "vdim")}, gate_cap=float(_need(d, "gate_cap", where)))
        if out.gate_cap <= 0:
            raise ConfigError(f"{where}gate_cap must be positive")
        return out

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: MemoryConfig

    @classmethod
    def from_dict(cls, d: dict, where: str) -> ParallelConfig:
        out = cls(AttentionConfig.from_dict(_need(d, "left", where), where + "left."), MemoryConfig.from_dict(_need(d, "right", where), where + "right."))
        if out.left.kv_from is not None:
            raise ConfigError(f"{where}left.kv_from: the attention of a parallel mixer has keys and values of its own")
        return out

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


MIXERS = {"attention": AttentionConfig, "parallel": ParallelConfig}


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    experts: int
    identity: int
    top: int
    groups: int
    keep: int
    scale: float

    def to_dict(self) -> dict:
        router = {"experts": self.experts, "identity": self.identity, "top": self.top, "groups": {"count": self.groups, "keep": self.keep}, "scale": self.scale}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": router}


def feed_forward_from_dict(d: dict | None, where: str) -> DenseConfig | ExpertsConfig | None:
    if d is None:
        return None
    kind = _need(d, "kind", where)
    if kind == "dense":
        return DenseConfig(_positive(d, "ff", where))
    if kind != "moe":
        raise ConfigError(f"{where}kind {kind!r} is not a feed-forward of this design ('dense' or 'moe')")
    r, at = _need(d, "router", where), where + "router."
    groups = r.get("groups")
    out = ExpertsConfig(
        ff=_positive(_need(d, "expert", where), "ff", where + "expert."), experts=_positive(r, "experts", at), identity=int(r.get("identity") or 0),
        top=_positive(r, "top", at), groups=_positive(groups, "count", at + "groups.") if groups else 1,
        keep=_positive(groups, "keep", at + "groups.") if groups else 1, scale=float(r.get("scale", 1.0)),
    )  # fmt: skip
    choices = out.experts + out.identity
    if out.identity < 0 or choices % out.groups or out.keep > out.groups:
        raise ConfigError(f"{at}groups must divide the experts and identity experts together, and keep at most count of them")
    if out.top > out.keep * (choices // out.groups):
        raise ConfigError(f"{at}top is more than the kept groups hold")
    return out


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: AttentionConfig | ParallelConfig
    mlp: DenseConfig | ExpertsConfig | None  # None: the layer has no feed-forward


@dataclass
class LatuzenConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    layers: list[LayerConfig]
    architectures: list[str] = field(default_factory=lambda: [ARCHITECTURE])
    raw: dict[str, Any] = field(default_factory=dict, repr=False)

    @property
    def architecture(self) -> str:
        return self.architectures[0]

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def max_position_embeddings(self) -> int:
        return 1 << 30  # the design names no longest sequence

    def __post_init__(self) -> None:
        for i, lc in enumerate(self.layers):
            if lc.type != "attention" or lc.mixer.kv_from is None:
                continue
            a, where = lc.mixer, f"layers[{i}].mixer.kv_from"
            src = self.layers[a.kv_from] if 0 <= a.kv_from < i else None
            if src is None or src.type != "attention" or src.mixer.kv_from is not None:
                raise ConfigError(f"{where} must name an earlier attention layer with keys and values of its own")
            if (src.mixer.kv_heads, src.mixer.dim, src.mixer.vdim) != (a.kv_heads, a.dim, a.vdim):
                raise ConfigError(f"{where} names a layer whose keys and values have another shape")

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> LatuzenConfig:
        layers = []
        for i, ld in enumerate(_need(d, "layers", "")):
            where = f"layers[{i}]."
            kind = _need(ld, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"{where}type {kind!r} is not a mixer of this design ({sorted(MIXERS)})")
            mixer = MIXERS[kind].from_dict(_need(ld, "mixer", where), where + "mixer.")
            layers.append(LayerConfig(kind, mixer, feed_forward_from_dict(ld.get("mlp"), where + "mlp.")))
        return cls(
            vocab_size=_positive(d, "vocab", ""), hidden_size=_positive(d, "width", ""), eps=float(_need(_need(d, "norm", ""), "eps", "norm.")),
            layers=layers, raw=dict(d),
        )  # fmt: skip

    def to_hf_dict(self) -> dict[str, Any]:
        return {
            "architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.eps},
            "layers": [{"type": lc.type, "mixer": lc.mixer.to_dict(), "mlp": lc.mlp.to_dict() if lc.mlp is not None else None} for lc in self.layers],
        }  # fmt: skip


def patterned(
    *, vocab: int, width: int, pattern: str, repeats: int, heads: int, kv_heads: int, dim: int, window: int, left_window: int, rot: RotationConfig,
    left_rot: RotationConfig, right_heads: int, right_dim: int, ff: int, experts: ExpertsConfig, gate_cap: float = 12.0, eps: float = 1e-6,
) -> LatuzenConfig:  # fmt: skip
    """A configuration whose layers follow ``pattern`` ``repeats`` times, two letters a layer.  The mixer: ``a`` attention, ``s`` attention over
    the keys and values of the ``a`` layer before it, ``p`` attention beside a matrix memory.  The feed-forward: ``d`` dense, ``e`` routed
    experts, ``-`` none.  What the named shapes below are made with."""
    layers: list[LayerConfig] = []
    own = None
    for i, (kind, ffn) in enumerate(zip(pattern[::2] * repeats, pattern[1::2] * repeats)):
        if kind == "a":
            own = i
        if kind == "p":
            left = AttentionConfig(heads, kv_heads, dim, dim, dim**-0.5, left_window, left_rot)
            mixer = ("parallel", ParallelConfig(left, MemoryConfig(right_heads, right_dim, right_dim, gate_cap)))
        else:
            mixer = ("attention", AttentionConfig(heads, kv_heads, dim, dim, dim**-0.5, window, rot, own if kind == "s" else None))
        layers.append(LayerConfig(*mixer, {"d": DenseConfig(ff), "e": experts, "-": None}[ffn]))
    return LatuzenConfig(vocab, width, eps, layers)


# Named shapes with random weights: a small one for demonstrations, and two with the width, depth and vocabulary of the 1B and 3B Llama
# shapes this engine is measured on (a dense feed-forward of that shape's flops; experts of which a token uses 4 with as many flops).
LATUZEN_PRESETS: dict[str, LatuzenConfig] = {
    "latuzen-tiny": patterned(
        vocab=256, width=80, pattern="adsepdse", repeats=1, heads=4, kv_heads=2, dim=32, window=40, left_window=24,
        rot=RotationConfig(24, 10000.0, YarnConfig(4.0, 64, 8.0, 1.0)), left_rot=RotationConfig(16, 10000.0), right_heads=2, right_dim=16, ff=128,
        experts=ExpertsConfig(ff=40, experts=6, identity=2, top=2, groups=2, keep=1, scale=1.5),
    ),
    "latuzen-1b": patterned(
        vocab=128256, width=2048, pattern="adsepdse", repeats=4, heads=32, kv_heads=8, dim=64, window=1024, left_window=1024,
        rot=RotationConfig(64, 500000.0, YarnConfig(8.0, 2048, 32.0, 1.0)), left_rot=RotationConfig(64, 500000.0), right_heads=16, right_dim=128,
        ff=8192, experts=ExpertsConfig(ff=1408, experts=32, identity=8, top=4, groups=4, keep=2, scale=2.5),
    ),
    "latuzen-3b": patterned(
        vocab=128256, width=3072, pattern="adsepdse", repeats=7, heads=24, kv_heads=8, dim=128, window=1024, left_window=1024,
        rot=RotationConfig(128, 500000.0, YarnConfig(8.0, 2048, 32.0, 1.0)), left_rot=RotationConfig(64, 500000.0), right_heads=24, right_dim=128,
        ff=8192, experts=ExpertsConfig(ff=1408, experts=32, identity=8, top=4, groups=4, keep=2, scale=2.5),
    ),
}  # fmt: skip
