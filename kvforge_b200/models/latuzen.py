"""The Latuzen decoder as a ``ModelSpec``: which parts, with which constants, under which tensor names.

Every layer is the parallel arrangement (``h = norm1(x)``, ``x += mixer(h) + ffn(h)``) with a layer norm that has weight and bias.  Its
mixer is grouped-query attention under a sliding window (queries and keys normed as one vector each, with biases, turned in split
pairs by YaRN-scaled frequencies), possibly over the keys and values of an earlier layer; or such attention (heads normed
one by one, turned in interleaved pairs, a sink whose score is zero) beside a matrix memory with exponential gates, as the mean of the
two normed results.  Its feed-forward is the dense gated one, or routed gated experts some of which hand their input on (softmax
scores, a correction that moves the choice alone, groups ranked by their best member, scaled weights), or absent.  Tensors
of layer ``i`` start with ``l<i>.``."""

from __future__ import annotations

from ..config.latuzen_config import AttentionConfig, DenseConfig, ExpertsConfig, LatuzenConfig, MemoryConfig, RotationConfig
from ..parts.base import PartSpec
from ..parts.model import LayerCall, LayerSpec, ModelSpec


def _rotary(head_dim: int, rot: RotationConfig | None, interleaved: bool) -> PartSpec | None:
    if rot is None:
        return None
    scaling = {"type": "yarn", **rot.scaling.to_dict()} if rot.scaling is not None else None
    return PartSpec("rotary", {"head_dim": head_dim, "rotary_dim": rot.dims, "theta": rot.base, "interleaved": interleaved, "scaling": scaling})


def _sizes(cfg: LatuzenConfig, a: AttentionConfig, interleaved: bool) -> dict:
    return {
        "hidden_size": cfg.hidden_size, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.vdim,
        "scale": a.scale, "window": a.window, "position": _rotary(a.dim, a.rot, interleaved),
    }  # fmt: skip


def _attention(cfg: LatuzenConfig, a: AttentionConfig, keep_window: int, keep_all: bool) -> PartSpec:
    params = {"qkv_bias": True, "joint_norm": {"eps": cfg.eps}, "gate": None, "shared_kv": a.kv_from is not None}
    return PartSpec("gated_attention", {**_sizes(cfg, a, False), **params, "keep_window": keep_window, "keep_all": keep_all})


def _left(cfg: LatuzenConfig, a: AttentionConfig) -> PartSpec:
    names = {
        "q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o", "q_norm.weight": "q.norm", "k_norm.weight": "k.norm",
    }  # fmt: skip
    return PartSpec("paged_attention", {**_sizes(cfg, a, True), "qk_norm": {"eps": cfg.eps}, "sink": "zero", "pad_heads": True, "names": names})


def _right(cfg: LatuzenConfig, r: MemoryConfig) -> PartSpec:
    return PartSpec(
        "matrix_memory",
        {"hidden_size": cfg.hidden_size, "num_heads": r.heads, "head_dim": r.dim, "v_head_dim": r.vdim, "gate_cap": r.gate_cap, "eps": cfg.eps},
    )


def _feed_forward(cfg: LatuzenConfig, m: DenseConfig | ExpertsConfig | None) -> PartSpec | None:
    if m is None:
        return None
    if isinstance(m, DenseConfig):
        names = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}
        return PartSpec("gated_mlp", {"hidden_size": cfg.hidden_size, "intermediate_size": m.ff, "activation": "silu", "names": names})
    return PartSpec(
        "routed_experts",
        {
            "hidden_size": cfg.hidden_size, "experts": m.experts, "identity": m.identity, "top": m.top, "intermediate_size": m.ff,
            "groups": m.groups, "keep": m.keep, "group_rank": "max", "correction": True, "score": "softmax", "normalize": False,
            "weight_scale": m.scale, "activation": "gated",
        },
    )  # fmt: skip


def latuzen_spec(cfg: LatuzenConfig) -> ModelSpec:
    def norm(name: str) -> dict:
        return {"dim": cfg.hidden_size, "eps": cfg.eps, "bias": True, "names": {"weight": name, "bias": f"{name}.b"}}

    # what a layer's cache has to keep for the layers that read it: the longest window among them, or every key
    longest: dict[int, int] = {}
    whole: set[int] = set()
    for lc in cfg.layers:
        source = lc.mixer.kv_from if lc.type == "attention" else None
        if source is None:
            continue
        if lc.mixer.window is None:
            whole.add(source)
        else:
            longest[source] = max(longest.get(source, 0), lc.mixer.window)
    layers, execution = [], []
    for i, lc in enumerate(cfg.layers):
        m = lc.mixer
        source = None
        if lc.type == "attention":
            source = m.kv_from
            keep = longest.get(i, 0) if m.window is not None else 0
            mixer = _attention(cfg, m, keep if keep > (m.window or 0) else 0, i in whole)
        else:
            mixer = PartSpec("parallel_mixers", {"hidden_size": cfg.hidden_size, "eps": cfg.eps, "branches": [("left", _left(cfg, m.left)), ("right", _right(cfg, m.right))]})
        block = PartSpec("parallel", {"norm": PartSpec("layernorm", norm("norm1")), "norm_name": "", "mixer": mixer, "ffn": _feed_forward(cfg, lc.mlp)})
        layers.append(LayerSpec(block=block, prefix=f"l{i}."))
        execution.append(LayerCall(i, kv_from=source))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=cfg.hidden_size,
        vocab_size=cfg.vocab_size,
        layers=layers,
        execution=execution,
        final_norm=PartSpec("layernorm", norm("norm")),
        final_norm_prefix="final.",
        embedding_name="embed",
        lm_head_name="head",
        ignore_suffixes=(),
        max_position_embeddings=cfg.max_position_embeddings,
    )
