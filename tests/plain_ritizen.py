"""A plain, slow implementation of the Ritizen decoder: whole sequences, no cache, no batching, one
function per mechanism, written from the design's equations.  It shares no code with the package and
is what the package's kernels are compared with.

Notation: ``T`` tokens, ``W`` model width, ``H`` heads, ``G`` key heads (or groups), ``dk`` / ``dv`` the
key and value sizes of a head.  Weights are a dict name -> tensor with the checkpoint's names; ``cfg``
is the parsed ``config.json``.  Everything runs in the dtype of the weights (float32 or float64) on
the CPU.
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


def rms_norm(x, weight, eps: float):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z**3)))


def softplus(z):
    """log(1 + e^z), without a clamp and without overflow."""
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(x, taps, bias):
    """``x [T, C]``, ``taps [C, n]`` whose last column multiplies the token itself; zeros before the start."""
    t, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x) + bias
    for back in range(n):
        rows = t - back
        if rows > 0:
            y[back:] += x[:rows] * taps[:, n - 1 - back]
    return y


# ---------------------------------------------------------------- attention


def whole_causal(t: int):
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    return j <= i


def chunked_causal(t: int, size: int):
    """A position sees itself and the earlier positions of its own chunk (positions ``c * size`` to ``c * size + size - 1``)."""
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    return (j <= i) & (i // size == j // size)


def keys_and_values(h, w, p: str, m: dict, eps: float):
    """(keys ``[T, G, dk]`` after their norm, values ``[T, G, dv]``) of a layer that projects its own."""
    t = h.shape[0]
    k, v = h @ w[p + "k"].T, h @ w[p + "v"].T
    if p + "k.b" in w:
        k, v = k + w[p + "k.b"], v + w[p + "v.b"]
    k = rms_norm(k, w[p + "k.norm"], eps)
    return k.reshape(t, m["kv_heads"], m["dim"]), v.reshape(t, m["kv_heads"], m["vdim"])


def attention(h, w, p: str, m: dict, eps: float, k, v):
    """Grouped-query attention over given keys and values.  The query rows of all heads are normed as one
    vector; nothing turns with the position; the gate has one number a head or one a channel, whichever
    the rows of its matrix say."""
    t = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = h @ w[p + "q"].T
    if p + "q.b" in w:
        q = q + w[p + "q.b"]
    q = rms_norm(q, w[p + "q.norm"], eps).reshape(t, H, dk)
    visible = chunked_causal(t, m["mask"]["size"]) if m.get("mask") else whole_causal(t)
    out = h.new_zeros(t, H, dv)
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T) * m["scale"]
        out[:, head] = torch.softmax(s.masked_fill(~visible, float("-inf")), dim=-1) @ v[:, g]
    gate = torch.sigmoid(h @ w[p + "g"].T)
    if gate.shape[1] == H:
        out = (out * gate[:, :, None]).reshape(t, H * dv)
    else:
        out = out.reshape(t, H * dv) * gate
    return out @ w[p + "o"].T


# ---------------------------------------------------------------- recurrences


def fixed_decay_walk(q, k, v, decay):
    """``S_t = decay_h S_(t-1) + k_t v_t^T``, ``o_t = S_t^T q_t``: ``[T, H, dk]`` twice and ``[T, H, dv]`` in, ``[T, H, dv]`` out."""
    t, H, dk = q.shape
    state = q.new_zeros(H, dk, v.shape[2])
    a = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    out = []
    for s in range(t):
        state = a * state + k[s][:, :, None] * v[s][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", state, q[s]))
    return torch.stack(out)


def lightning_attention(h, w, p: str, m: dict, eps: float):
    t = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(t, H, dk)
    k = silu(h @ w[p + "k"].T).reshape(t, H, dk)
    v = silu(h @ w[p + "v"].T).reshape(t, H, dv)
    o = fixed_decay_walk(q, k, v, m["decay"]).reshape(t, H * dv)
    o = rms_norm(o, w[p + "norm"], eps) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def state_space_walk(x, b, c, dt, a_log, skip):
    """``S_t = exp(-exp(a_log_h) dt) S_(t-1) + dt B x^T``, ``y_t = S_t^T C + skip_h x``; ``x [T, H, dv]``, ``b`` and ``c``
    ``[T, G, N]`` (head ``h`` takes group ``h // (H / G)``), ``dt [T, H]``."""
    t, H, dv = x.shape
    G, N = b.shape[1], b.shape[2]
    of = torch.arange(H) // (H // G)
    state = x.new_zeros(H, N, dv)
    out = []
    for s in range(t):
        a = torch.exp(-torch.exp(a_log) * dt[s])[:, None, None]
        state = a * state + dt[s][:, None, None] * b[s][of][:, :, None] * x[s][:, None, :]
        out.append(torch.einsum("hnv,hn->hv", state, c[s][of]) + skip[:, None] * x[s])
    return torch.stack(out)


def grouped_rms_norm(y, weight, parts: int, eps: float):
    """Each of ``parts`` equal stretches of the last axis is divided by its own root mean square."""
    t, c = y.shape
    u = y.reshape(t, parts, c // parts)
    u = u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)
    return u.reshape(t, c) * weight


def mamba2(h, w, p: str, m: dict, eps: float):
    t = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    y = h @ w[p + "in"].T
    z, xbc, dt = y[:, :inner], y[:, inner : 2 * inner + 2 * G * N], y[:, 2 * inner + 2 * G * N :]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, b, c = xbc[:, :inner], xbc[:, inner : inner + G * N], xbc[:, inner + G * N :]
    dt = softplus(dt + w[p + "dt_bias"])
    o = state_space_walk(x.reshape(t, H, dv), b.reshape(t, G, N), c.reshape(t, G, N), dt, w[p + "A_log"], w[p + "D"])
    o = o.reshape(t, inner) * silu(z)
    return grouped_rms_norm(o, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward


def feed_forward(h, w, p: str):
    u = gelu_tanh(h @ w[p + "up"].T + w[p + "up.b"])
    return u @ w[p + "down"].T + w[p + "down.b"]


# ---------------------------------------------------------------- the model


def embed(cfg, w, tokens):
    ids = torch.as_tensor(tokens, dtype=torch.long)
    return w["embed"][ids] + w["pos"][: len(ids)]


def residual_after_every_layer(cfg, w, tokens) -> list[torch.Tensor]:
    eps = cfg["norm"]["eps"]
    x = embed(cfg, w, tokens)
    out = []
    kept = {}  # layer -> (keys, values)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        if layer["type"] == "attention":
            kept[i] = kept[m["kv_from"]] if m.get("kv_from") is not None else keys_and_values(x, w, p, m, eps)
            y = attention(x, w, p, m, eps, *kept[i])
        elif layer["type"] == "parallel":
            left = m["left"]
            kept[i] = keys_and_values(x, w, p + "left.", left, eps)
            y = m["left_scale"] * attention(x, w, p + "left.", left, eps, *kept[i])
            y = y + m["right_scale"] * lightning_attention(x, w, p + "right.", m["right"], eps)
        else:
            y = mamba2(x, w, p, m, eps)
        x = x + rms_norm(y, w[f"l{i}.norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + rms_norm(feed_forward(x, w, f"l{i}.mlp."), w[f"l{i}.norm2"], eps)
        out.append(x)
    return out


def logits(cfg, w, tokens) -> torch.Tensor:
    x = residual_after_every_layer(cfg, w, tokens)[-1]
    return rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T


def greedy(cfg, w, prompt, n_new: int) -> list[int]:
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(logits(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt) :]
