"""The Ritizen decoder as a ``ModelSpec``: which parts, with which constants, under which tensor names.

The embedding's row and a learned vector of the position are the stream.  Every layer norms its sublayers' results only
(``x += norm1(mixer(x))``, ``x += norm2(ffn(x))``).  Its mixer is grouped-query attention without rotation (queries and keys
normed as one vector each, a gate a head), possibly over the keys and values of an earlier layer; a state space whose step
size follows the token; or chunked attention (with biases and a gate a channel) and lightning attention side by side,
each times a constant.  Its feed-forward is the plain one with biases and the tanh form of gelu, or absent.  The logits are
products with the embedding's table.  Tensors of layer ``i`` start with ``l<i>.``."""

from __future__ import annotations

from ..config.ritizen_config import AttentionConfig, LightningConfig, Mamba2Config, RitizenConfig
from ..parts.base import PartSpec
from ..parts.model import LayerCall, LayerSpec, ModelSpec


def _attention(cfg: RitizenConfig, a: AttentionConfig, gate: str, bias: bool, keep_all: bool) -> PartSpec:
    return PartSpec(
        "gated_attention",
        {
            "hidden_size": cfg.hidden_size, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.vdim,
            "scale": a.scale, "chunk": a.chunk, "qkv_bias": bias, "joint_norm": {"eps": cfg.eps}, "gate": gate,
            "shared_kv": a.kv_from is not None, "keep_all": keep_all,
        },
    )  # fmt: skip


def _lightning(cfg: RitizenConfig, r: LightningConfig) -> PartSpec:
    return PartSpec(
        "retention",
        {
            "hidden_size": cfg.hidden_size, "num_heads": r.heads, "head_dim": r.dim, "v_head_dim": r.vdim, "decay": list(r.decay),
            "eps": cfg.eps, "key_scale": 1.0, "activation": "silu", "norm": "joint", "gate": "sigmoid",
        },
    )  # fmt: skip


def _state_space(cfg: RitizenConfig, m: Mamba2Config) -> PartSpec:
    return PartSpec(
        "state_space",
        {
            "hidden_size": cfg.hidden_size, "num_heads": m.heads, "v_head_dim": m.vdim, "state_dim": m.state, "groups": m.groups,
            "conv": m.conv, "norm_groups": m.norm_groups, "eps": cfg.eps,
        },
    )  # fmt: skip


def ritizen_spec(cfg: RitizenConfig) -> ModelSpec:
    norm = {"dim": cfg.hidden_size, "eps": cfg.eps, "centred": False}
    # a chunked layer whose keys a later layer reads beyond its chunks keeps them all
    read_whole = set()
    for lc in cfg.layers:
        a = lc.attention
        if a is not None and a.kv_from is not None and cfg.layers[a.kv_from].attention.chunk not in (None, a.chunk):
            read_whole.add(a.kv_from)
    layers, execution = [], []
    for i, lc in enumerate(cfg.layers):
        m = lc.mixer
        if lc.type == "attention":
            mixer = _attention(cfg, m, "head", False, i in read_whole)
        elif lc.type == "parallel":
            mixer = PartSpec(
                "summed_mixers",
                {
                    "hidden_size": cfg.hidden_size,
                    "branches": [
                        ("left", _attention(cfg, m.left, "channel", True, i in read_whole), m.left_scale),
                        ("right", _lightning(cfg, m.right), m.right_scale),
                    ],
                },
            )
        else:
            mixer = _state_space(cfg, m)
        ffn = None
        if lc.ff is not None:
            ffn = PartSpec("plain_mlp", {"hidden_size": cfg.hidden_size, "intermediate_size": lc.ff, "activation": "gelu_tanh", "bias": True})
        block = PartSpec("postnorm", {"norm": PartSpec("layernorm", norm), "mixer": mixer, "ffn": ffn})
        layers.append(LayerSpec(block=block, prefix=f"l{i}."))
        execution.append(LayerCall(i, kv_from=lc.attention.kv_from if lc.attention is not None else None))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=cfg.hidden_size,
        vocab_size=cfg.vocab_size,
        layers=layers,
        execution=execution,
        final_norm=PartSpec("layernorm", {**norm, "names": {"weight": "norm"}}),
        final_norm_prefix="final.",
        tie_word_embeddings=True,
        embedding_name="embed",
        input_position=PartSpec("learned", {"rows": cfg.max_position_embeddings, "hidden_size": cfg.hidden_size, "names": {"weight": "pos"}}),
        input_position_prefix="",
        ignore_suffixes=(),
        max_position_embeddings=cfg.max_position_embeddings,
    )
