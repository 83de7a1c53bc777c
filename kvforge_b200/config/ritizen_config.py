"""Typed configuration of the Ritizen decoder, read from its ``config.json``.

The file gives every size and every constant that differs between models of the design::

    {"architecture": "Ritizen", "vocab": V, "width": W, "max_positions": P, "norm": {"eps": e},
     "layers": [{"type": "attention" | "parallel" | "mamba2", "mixer": {...}, "mlp": {"kind": "dense", "ff": F} | null}, ...]}

An ``attention`` mixer: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale`` and, in a layer that uses an earlier layer's keys
and values, ``kv_from``.  A ``parallel`` mixer: ``left`` (the same, with ``mask.size``: the positions of a chunk), ``right``
(``heads``, ``dim``, ``vdim``, ``decay``: one number a head), ``left_scale``, ``right_scale``.  A ``mamba2`` mixer: ``heads``,
``vdim``, ``state``, ``groups``, ``conv`` (taps), ``norm_groups``.  Nothing here has a default that stands for a size.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from .model_config import ConfigError

ARCHITECTURE = "Ritizen"


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
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int | None = None
    kv_from: int | None = None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> AttentionConfig:
        mask, source = d.get("mask"), d.get("kv_from")
        out = cls(
            **{k: _positive(d, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}, scale=float(_need(d, "scale", where)),
            chunk=_positive(mask, "size", where + "mask.") if mask else None, kv_from=int(source) if source is not None else None,
        )  # fmt: skip
        if out.heads % out.kv_heads:
            raise ConfigError(f"{where}heads must be a multiple of kv_heads")
        return out

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]

    @classmethod
    def from_dict(cls, d: dict, where: str) -> LightningConfig:
        out = cls(**{k: _positive(d, k, where) for k in ("heads", "dim", "vdim")}, decay=tuple(float(a) for a in _need(d, "decay", where)))
        if len(out.decay) != out.heads:
            raise ConfigError(f"{where}decay must hold one number per head")
        return out

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: LightningConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d: dict, where: str) -> ParallelConfig:
        out = cls(
            AttentionConfig.from_dict(_need(d, "left", where), where + "left."), LightningConfig.from_dict(_need(d, "right", where), where + "right."),
            float(_need(d, "left_scale", where)), float(_need(d, "right_scale", where)),
        )  # fmt: skip
        if out.left.kv_from is not None:
            raise ConfigError(f"{where}left.kv_from: the attention of a parallel mixer has keys and values of its own")
        return out

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale, "right_scale": self.right_scale}


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_dict(cls, d: dict, where: str) -> Mamba2Config:
        out = cls(**{k: _positive(d, k, where) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")})
        if out.heads % out.groups:
            raise ConfigError(f"{where}heads must be a multiple of groups")
        if (out.heads * out.vdim) % out.norm_groups:
            raise ConfigError(f"{where}norm_groups must divide heads * vdim")
        return out

    def to_dict(self) -> dict:
        return {k: getattr(self, k) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}


MIXERS = {"attention": AttentionConfig, "parallel": ParallelConfig, "mamba2": Mamba2Config}


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: AttentionConfig | ParallelConfig | Mamba2Config
    ff: int | None  # None: the layer has no feed-forward

    @property
    def attention(self) -> AttentionConfig | None:
        """The layer's attention, if it has one."""
        return self.mixer if self.type == "attention" else self.mixer.left if self.type == "parallel" else None


def _ff(mlp: dict | None, where: str) -> int | None:
    if mlp is None:
        return None
    if _need(mlp, "kind", where) != "dense":
        raise ConfigError(f"{where}kind {mlp['kind']!r} is not a feed-forward of this design (only 'dense')")
    return _positive(mlp, "ff", where)


@dataclass
class RitizenConfig:
    vocab_size: int
    hidden_size: int
    max_position_embeddings: int
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

    def __post_init__(self) -> None:
        for i, lc in enumerate(self.layers):
            a = lc.attention
            if a is None or a.kv_from is None:
                continue
            where = f"layers[{i}].mixer.kv_from"
            src = self.layers[a.kv_from].attention if 0 <= a.kv_from < i else None
            if src is None or src.kv_from is not None:
                raise ConfigError(f"{where} must name an earlier layer with keys and values of its own")
            if (src.kv_heads, src.dim, src.vdim) != (a.kv_heads, a.dim, a.vdim):
                raise ConfigError(f"{where} names a layer whose keys and values have another shape")

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> RitizenConfig:
        layers = []
        for i, ld in enumerate(_need(d, "layers", "")):
            where = f"layers[{i}]."
            kind = _need(ld, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"{where}type {kind!r} is not a mixer of this design ({sorted(MIXERS)})")
            layers.append(LayerConfig(kind, MIXERS[kind].from_dict(_need(ld, "mixer", where), where + "mixer."), _ff(ld.get("mlp"), where + "mlp.")))
        return cls(
            vocab_size=_positive(d, "vocab", ""), hidden_size=_positive(d, "width", ""), max_position_embeddings=_positive(d, "max_positions", ""),
            eps=float(_need(_need(d, "norm", ""), "eps", "norm.")), layers=layers, raw=dict(d),
        )  # fmt: skip

    def to_hf_dict(self) -> dict[str, Any]:
        return {
            "architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "max_positions": self.max_position_embeddings,
            "norm": {"eps": self.eps},
            "layers": [
                {"type": lc.type, "mixer": lc.mixer.to_dict(), "mlp": {"kind": "dense", "ff": lc.ff} if lc.ff is not None else None} for lc in self.layers
            ],
        }  # fmt: skip


def patterned(
    *, vocab: int, width: int, max_positions: int, pattern: str, repeats: int, heads: int, kv_heads: int, dim: int, chunk: int,
    right_heads: int, right_dim: int, ssm_heads: int, ssm_dim: int, state: int, groups: int, norm_groups: int, ff: int, conv: int = 4,
    eps: float = 1e-6,
) -> RitizenConfig:  # fmt: skip
    """A configuration whose layers follow ``pattern`` ``repeats`` times, a letter a layer: ``a`` attention, ``s`` attention over
    the keys and values of the ``a`` layer before it, ``m`` a state space, ``p`` chunked attention beside lightning attention;
    an upper-case letter is a layer without a feed-forward.  What the named shapes below are made with.  Lightning heads
    decay by ``1 - 2^-(3 + h)``."""
    right = LightningConfig(right_heads, right_dim, right_dim, tuple(1.0 - 2.0 ** -(3 + h % 8) for h in range(right_heads)))
    layers: list[LayerConfig] = []
    own = None
    for i, letter in enumerate(pattern * repeats):
        kind, source = letter.lower(), None
        if kind == "a":
            own = i
        if kind == "s":
            source = own
        attn = AttentionConfig(heads, kv_heads, dim, dim, dim**-0.5, chunk if kind == "p" else None, source)
        mixer = {
            "a": ("attention", attn), "s": ("attention", attn), "p": ("parallel", ParallelConfig(attn, right, 0.75, 0.5)),
            "m": ("mamba2", Mamba2Config(ssm_heads, ssm_dim, state, groups, conv, norm_groups)),
        }[kind]  # fmt: skip
        layers.append(LayerConfig(*mixer, None if letter.isupper() else ff))
    return RitizenConfig(vocab, width, max_positions, eps, layers)


# Named shapes with random weights: a small one for demonstrations, and two with the width, depth and vocabulary of the 1B
# and 3B Llama shapes this engine is measured on (the plain feed-forward's two matrices are as many numbers as that
# shape's gated three; the state-space layers, whose projections are twice as wide as an attention layer's, have one too).
RITIZEN_PRESETS: dict[str, RitizenConfig] = {
    "ritizen-tiny": patterned(
        vocab=256, width=96, max_positions=512, pattern="asMp", repeats=1, heads=4, kv_heads=2, dim=32, chunk=24, right_heads=2, right_dim=16,
        ssm_heads=4, ssm_dim=16, state=24, groups=2, norm_groups=2, ff=128, conv=3,
    ),
    "ritizen-1b": patterned(
        vocab=128256, width=2048, max_positions=16384, pattern="asmp", repeats=4, heads=32, kv_heads=8, dim=64, chunk=1024, right_heads=16,
        right_dim=128, ssm_heads=64, ssm_dim=64, state=128, groups=1, norm_groups=1, ff=12288,
    ),
    "ritizen-3b": patterned(
        vocab=128256, width=3072, max_positions=16384, pattern="asmp", repeats=7, heads=24, kv_heads=8, dim=128, chunk=1024, right_heads=24,
        right_dim=128, ssm_heads=96, ssm_dim=64, state=128, groups=2, norm_groups=2, ff=12288,
    ),
}  # fmt: skip
