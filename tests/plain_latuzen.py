"""A plain, slow implementation of the Latuzen decoder: whole sequences, no cache, no batching, one function per
mechanism, written from the design's equations.  It shares no code with the package and is what the package's kernels
are compared with.

Notation: ``T`` tokens, ``W`` model width, ``H`` heads, ``G`` key heads, ``dk`` / ``dv`` the key and value sizes of a head,
``E`` experts, ``I`` identity experts.  Weights are a dict name -> tensor with the checkpoint's names; ``cfg`` is the
parsed ``config.json``.  Everything runs in the dtype of the weights (float32 or float64) on the CPU.
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch


# ---------------------------------------------------------------- reading a folder


def read_folder(folder, dtype=torch.float64):
    """(config dict, weights dict) of a model folder; floats widened to ``dtype``."""
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8 : 8 + n])
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "F64": torch.float64}
    weights = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        t = torch.frombuffer(bytearray(raw[8 + n + a : 8 + n + b]), dtype=kinds[info["dtype"]]).reshape(info["shape"])
        weights[name] = t.to(dtype) if t.is_floating_point() else t
    return cfg, weights


# ---------------------------------------------------------------- small pieces


def layer_norm(x, weight, bias, eps: float):
    """Mean taken off, divided by the root of the mean squared deviation (plus eps), weight and bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def unit_rms(x, eps: float):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def log_sigmoid(z):
    """-log(1 + e^-z) without overflow."""
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


# ---------------------------------------------------------------- rotation


def frequencies(rot: dict) -> list[float]:
    """One frequency a pair of dims, with the blend of scaled and plain frequencies where ``scaling`` is given."""
    dims, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return plain

    def dim_of(turns):  # the (fractional) dim whose wave turns so many times within the original context
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(dim_of(s["fast"])), 0), min(math.ceil(dim_of(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out


def rotation_size(rot: dict) -> float:
    """What cosine and sine are multiplied by."""
    return 0.1 * math.log(rot["scaling"]["factor"]) + 1.0 if rot.get("scaling") else 1.0


def rotate(x, rot: dict, interleaved: bool):
    """``x [T, heads, d]`` at positions 0 .. T-1; the dims beyond ``rot['dims']`` pass."""
    t, dims = x.shape[0], rot["dims"]
    half = dims // 2
    angle = torch.arange(t, dtype=x.dtype)[:, None] * torch.tensor(frequencies(rot), dtype=x.dtype)[None, :]
    c, s = (torch.cos(angle) * rotation_size(rot))[:, None, :], (torch.sin(angle) * rotation_size(rot))[:, None, :]
    out = x.clone()
    first = slice(0, dims, 2) if interleaved else slice(0, half)
    second = slice(1, dims, 2) if interleaved else slice(half, dims)
    u, v = x[..., first], x[..., second]
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


# ---------------------------------------------------------------- attention


def window_mask(t: int, size: int):
    """[T, T], true where the query (row) sees the key (column): itself and the ``size - 1`` tokens before it."""
    back = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return (back >= 0) & (back < size)


def attend(q, k, v, scale: float, visible, sink: bool):
    """``q [T, H, dk]``, ``k [T, G, dk]``, ``v [T, G, dv]`` -> ``[T, H, dv]``; ``sink``: one is added to the denominator."""
    t, H, _ = q.shape
    G = k.shape[1]
    out = q.new_zeros(t, H, v.shape[2])
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T * scale).masked_fill(~visible, float("-inf"))
        top = s.max(-1, keepdim=True).values
        if sink:
            top = torch.clamp(top, min=0.0)
        e = torch.exp(s - top)
        total = e.sum(-1, keepdim=True) + (torch.exp(-top) if sink else 0.0)
        out[:, head] = e / total @ v[:, g]
    return out


def keys_and_values(h, w, p: str, m: dict, eps: float):
    """Keys and values of an ``attention`` layer that projects its own: biases, the keys' norm over all heads at once, rotation."""
    t = h.shape[0]
    k = unit_rms(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]
    v = h @ w[p + "v"].T + w[p + "v.b"]
    return rotate(k.reshape(t, m["kv_heads"], m["dim"]), m["rot"], False), v.reshape(t, m["kv_heads"], m["vdim"])


def jointly_normed_attention(h, w, p: str, m: dict, eps: float, k, v):
    t = h.shape[0]
    q = unit_rms(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]
    q = rotate(q.reshape(t, m["heads"], m["dim"]), m["rot"], False)
    o = attend(q, k, v, m["scale"], window_mask(t, m["mask"]["size"]), False)
    return o.reshape(t, -1) @ w[p + "o"].T


def left_keys_and_values(h, w, p: str, m: dict, eps: float):
    t = h.shape[0]
    k = unit_rms((h @ w[p + "k"].T).reshape(t, m["kv_heads"], m["dim"]), eps) * w[p + "k.norm"]
    return rotate(k, m["rot"], True), (h @ w[p + "v"].T).reshape(t, m["kv_heads"], m["vdim"])


def sink_attention(h, w, p: str, m: dict, eps: float):
    t = h.shape[0]
    k, v = left_keys_and_values(h, w, p, m, eps)
    q = unit_rms((h @ w[p + "q"].T).reshape(t, m["heads"], m["dim"]), eps) * w[p + "q.norm"]
    o = attend(rotate(q, m["rot"], True), k, v, m["scale"], window_mask(t, m["mask"]["size"]), True)
    return o.reshape(t, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- matrix memory


def matrix_memory_walk(q, k, v, log_in, log_keep):
    """``q``, ``k`` ``[T, H, dk]``, ``v [T, H, dv]``, logarithms of the input and forget gates ``[T, H]`` -> ``[T, H, dv]``.  The state
    and the key sum are kept relative to ``e^top``, ``top`` the running maximum, which starts at zero."""
    t, H, dk = q.shape
    state, total, top = q.new_zeros(H, dk, v.shape[2]), q.new_zeros(H, dk), q.new_zeros(H)
    out = []
    for s in range(t):
        new_top = torch.maximum(log_keep[s] + top, log_in[s])
        keep, add = torch.exp(log_keep[s] + top - new_top), torch.exp(log_in[s] - new_top)
        state = keep[:, None, None] * state + add[:, None, None] * k[s][:, :, None] * v[s][:, None, :]
        total = keep[:, None] * total + add[:, None] * k[s]
        top = new_top
        size = torch.maximum((total * q[s]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out.append(torch.einsum("hkv,hk->hv", state, q[s]) / size[:, None])
    return torch.stack(out)


def memory_gates(h, w, p: str, cap: float):
    """(log input gate, log forget gate), ``[T, H]`` each."""
    log_in = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    return log_in, log_sigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))


def matrix_memory(h, w, p: str, m: dict, eps: float):
    t, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(t, H, dk) * dk**-0.5
    k, v = (h @ w[p + "k"].T).reshape(t, H, dk), (h @ w[p + "v"].T).reshape(t, H, dv)
    o = unit_rms(matrix_memory_walk(q, k, v, *memory_gates(h, w, p, m["gate_cap"])), eps)
    return (o.reshape(t, H * dv) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(h, w, p: str, m: dict, eps: float):
    left = unit_rms(sink_attention(h, w, p + "left.", m["left"], eps), eps) * w[p + "left.out"]
    right = unit_rms(matrix_memory(h, w, p + "right.", m["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (left + right)


# ---------------------------------------------------------------- feed-forward


def route(h, w, p: str, r: dict):
    """(chosen ``[T, top]``, their weights): the choice is made on the softmax's scores plus the correction, inside the best groups."""
    score = torch.softmax(h @ w[p + "router"].T, dim=-1)
    pick = score + w[p + "correction"]
    groups, keep = r["groups"]["count"], r["groups"]["keep"]
    ids, weights = [], []
    for s, c in zip(score.tolist(), pick.tolist()):
        size = len(c) // groups
        best = sorted(range(groups), key=lambda g: -max(c[g * size : (g + 1) * size]))[:keep]
        able = [e for e in range(len(c)) if e // size in best]
        chosen = sorted(able, key=lambda e: -c[e])[: r["top"]]
        ids.append(chosen)
        weights.append([s[e] * r["scale"] for e in chosen])
    return ids, torch.tensor(weights, dtype=h.dtype)


def routed_experts(h, w, p: str, m: dict):
    r = m["router"]
    ids, weights = route(h, w, p, r)
    out = torch.zeros_like(h)
    for t, chosen in enumerate(ids):
        for e, weight in zip(chosen, weights[t]):
            y = h[t] if e >= r["experts"] else gated_ff(h[t], *(w[f"{p}e{e}.{n}"] for n in ("gate", "up", "down")))
            out[t] += weight * y
    return out


def feed_forward(h, w, p: str, m: dict):
    if m["kind"] == "moe":
        return routed_experts(h, w, p, m)
    return gated_ff(h, w[p + "gate"], w[p + "up"], w[p + "down"])


# ---------------------------------------------------------------- the model


def residual_after_every_layer(cfg, w, tokens) -> list[torch.Tensor]:
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    out, kept = [], {}  # kept: layer -> (keys, values)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        if layer["type"] == "attention":
            kept[i] = kept[m["kv_from"]] if m.get("kv_from") is not None else keys_and_values(h, w, p + "mix.", m, eps)
            y = jointly_normed_attention(h, w, p + "mix.", m, eps, *kept[i])
        else:
            y = side_by_side(h, w, p + "mix.", m, eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, w, p + "mlp.", layer["mlp"])
        x = x + y
        out.append(x)
    return out


def logits(cfg, w, tokens) -> torch.Tensor:
    x = residual_after_every_layer(cfg, w, tokens)[-1]
    return layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"]) @ w["head"].T


def greedy(cfg, w, prompt, n_new: int) -> list[int]:
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(logits(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt) :]
