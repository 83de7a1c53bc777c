"""Grouped-query attention whose query rows (and key rows) are normed as one vector and whose result may be gated.

Per layer ``q = W_q x + b_q``, ``k = W_k x + b_k``, ``v = W_v x + b_v`` (the biases are optional); q and k are RMS-normed as
one vector each (all heads together), with weights as wide as the projections; then the first dims of every head may turn
with the position.  Attention sees every earlier key, a sliding window of them, or the keys of the query's own chunk.  The
result may be multiplied by ``sigmoid(W_g x)``, one number a head or one a channel, before the output projection.  A layer may
use the keys and values of an earlier layer (as that layer's cache holds them) with queries of its own.

The input projections (q, k, v and the gate) are one product.  Heads whose size is no multiple of 8 are padded with zeros
when the tensors are bound: zeros change neither a norm's sum nor a score nor, through zero columns of the output
projection, the result.
"""

from __future__ import annotations

import torch

from .. import ops
from .attention import PagedAttention, pad_head_rows
from .base import CacheNeed, WeightDecl, register_mixer
from .projection import PART_ROWS, project


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def stack_rows(mats: list[torch.Tensor]) -> tuple[torch.Tensor, list[int]]:
    """The matrices one below the other, each from a multiple of 8 rows on, and where each begins; the whole is a
    multiple of 8 rows long (rows of zeros between and after)."""
    rows, offs, at = [], [], 0
    for t in mats:
        offs.append(at)
        rows.append(t)
        pad = _pad8(t.shape[0]) - t.shape[0]
        if pad:
            rows.append(torch.zeros((pad, t.shape[1]), dtype=t.dtype, device=t.device))
        at += t.shape[0] + pad
    return torch.cat(rows, dim=0).contiguous(), offs


@register_mixer("gated_attention")
class GatedAttention(PagedAttention):
    """params: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``; optional ``v_head_dim``, ``scale``, ``window`` or
    ``chunk``, ``position`` (a rotation with any magnitude) and ``keep_window`` (as ``paged_attention``), ``qkv_bias`` (tensors ``q.b``, ``k.b``, ``v.b``), ``joint_norm`` (``{"eps": e}``: tensors
    ``q.norm``, ``k.norm``; ``None``: no norm), ``gate`` (``"head"``, ``"channel"`` or ``None``; tensor ``g``), ``shared_kv`` (keys and
    values are an earlier layer's: no tensors of its own for them) and ``keep_all`` (the cache keeps every key although
    this layer's queries do not see them all: a later layer that reads this cache does).  Other tensors: ``q``, ``k``, ``v``, ``o``.

    Besides ``forward`` it has the open form that ``summed_mixers`` takes: ``take_input`` / ``take_output`` hand the input and
    output matrices over, and ``mix`` computes what lies between the two products."""

    def __init__(self, params, prefix=""):
        p = dict(params)
        p["pad_heads"] = True
        super().__init__(p, prefix)
        self.params = dict(params)
        self.qkv_bias = bool(p.get("qkv_bias", False))
        jn = p.get("joint_norm")
        self.norm_eps = float(jn["eps"]) if jn else None
        self.out_gate = p.get("gate")
        if self.out_gate not in (None, "head", "channel"):
            raise ValueError("gate is 'head', 'channel' or None")
        self.shared_kv = bool(p.get("shared_kv", False))
        self.keep_all = bool(p.get("keep_all", False))
        self.own_kv = 0 if self.shared_kv else self.nkv
        if self.taps or self.qk_eps is not None or self.bias_shape or self.softcap or self.has_sink or self.value_mix:
            raise ValueError("gated_attention has no convolution, per-head norm, bias on scores, cap, sink or mixed values")
        self.qkv_dim = self.q_dim + self.own_kv * (self.d + self.dv)

    @classmethod
    def weight_decls(cls, params):
        h, nh, nkv, d = (int(params[k]) for k in ("hidden_size", "num_heads", "num_kv_heads", "head_dim"))
        dv = int(params.get("v_head_dim") or d)
        sizes = {"q": nh * d} if params.get("shared_kv") else {"q": nh * d, "k": nkv * d, "v": nkv * dv}
        out = {name: WeightDecl((n, h)) for name, n in sizes.items()}
        out["o"] = WeightDecl((h, nh * dv))
        if params.get("qkv_bias"):
            out.update({f"{name}.b": WeightDecl((n,), kind="vector", init="zeros") for name, n in sizes.items()})
        if params.get("joint_norm"):
            out.update({f"{name}.norm": WeightDecl((n,), kind="vector", init="ones") for name, n in sizes.items() if name != "v"})
        gate = params.get("gate")
        if gate:
            out["g"] = WeightDecl((nh if gate == "head" else nh * dv, h))
        return out

    def cache_need(self) -> CacheNeed:
        if self.keep_all:
            return CacheNeed("full", self.nkv, self.d, None, None if self.dv == self.d else self.dv)
        return super().cache_need()

    def bind(self, weights, rt):
        self.rt = rt
        nh, kv, d, dv = self.nh, self.own_kv, self.d, self.dv

        def heads(name: str, n: int, true: int, padded: int):
            return pad_head_rows(weights[name], n, true, padded)

        qkv = [heads("q", nh, self.d_true, d)]
        if kv:
            qkv += [heads("k", kv, self.d_true, d), heads("v", kv, self.dv_true, dv)]
        mats = [torch.cat(qkv, dim=0) if len(qkv) > 1 else qkv[0]]
        if self.out_gate:
            mats.append(weights["g"] if self.out_gate == "head" else heads("g", nh, self.dv_true, dv))
        self.w_in, offs = stack_rows(mats)
        self.in_dim = self.w_in.shape[0]
        self.gate_off = offs[1] if self.out_gate else None
        self.gate_dim = nh if self.out_gate == "head" else self.o_dim
        self.w_o = pad_head_rows(weights["o"].t().contiguous(), nh, self.dv_true, dv).t().contiguous() if dv != self.dv_true else weights["o"].contiguous()
        self.bias_vec = None
        if self.qkv_bias:
            b = [heads("q.b", nh, self.d_true, d)] + ([heads("k.b", kv, self.d_true, d), heads("v.b", kv, self.dv_true, dv)] if kv else [])
            self.bias_vec = torch.cat(b).contiguous()
        self.q_w = self.k_w = None
        if self.norm_eps is not None:
            self.q_w = heads("q.norm", nh, self.d_true, d).contiguous()
            self.k_w = heads("k.norm", kv, self.d_true, d).contiguous() if kv else None
        self._bind_position()
        self._bind_attention()

    # ------------------------------------------------------------------ between the two products
    open_form = True

    def take_input(self) -> torch.Tensor:
        w, self.w_in = self.w_in, None
        return w

    def take_output(self) -> torch.Tensor:
        w, self.w_o = self.w_o, None
        return w

    def mix(self, ctx, y: torch.Tensor, cache, out: torch.Tensor, mult: float = 1.0, parts=None) -> None:
        """``y [N, in_dim]``: the input product's rows (or room for them, when they still are the slices ``parts``);
        ``out [N, inner_width]`` gets ``mult`` times what the output projection multiplies."""
        if cache is None or cache.k is None:
            raise RuntimeError("gated_attention needs a cache")
        if cache.writable == self.shared_kv:
            raise RuntimeError("a layer with keys and values of its own writes its cache; one that shares another's only reads it")
        rt, n = self.rt, y.shape[0]
        own = self.own_kv > 0
        ops.joint_norm_cache(
            y, parts, self.bias_vec, self.q_w, self.k_w, self.nh * self.d_true, max(1, self.own_kv * self.d_true), self.norm_eps or 0.0,
            ctx.slot_mappings[cache.group] if own else None, cache.k if own else None, cache.v if own else None,
            self.nh, self.own_kv, self.d, self.dv, ctx.block_size, rt.err, positions=ctx.positions, inv_freq=self.inv_freq,
            interleaved=self.interleaved, magnitude=self.magnitude,
        )  # fmt: skip
        plain = self.out_gate is None and mult == 1.0 and out.is_contiguous()
        heads_out = out if plain else rt.buf("attn.out", n, self.o_dim)
        self.attend(ctx, y, y.stride(0), heads_out, cache)
        if plain:
            return
        if self.out_gate is None:
            raise RuntimeError("a result without a gate is neither scaled nor written into part of a wider row")
        ops.output_gate(heads_out, y[:, self.gate_off : self.gate_off + self.gate_dim], out, self.nh, self.dv, mult)

    def forward(self, ctx, x: torch.Tensor, cache) -> torch.Tensor:
        rt, n = self.rt, x.shape[0]
        y = rt.buf("gattn.in", n, self.in_dim)
        parts = None
        if ops.skinny_ok(x, self.w_in):
            splits = ops.skinny_splits(self.in_dim, self.hidden, n)
            if splits > 1:  # decode: slices of K in parallel, summed where the rows are normed
                parts = ops.Partials(rt.buf("gattn.in_part", splits * n, self.in_dim, torch.float32, cap=PART_ROWS).view(splits, n, self.in_dim))
                ops.gemm_skinny(x, self.w_in, parts)
            else:
                ops.gemm_skinny(x, self.w_in, y)
        else:
            ops.linear(x, self.w_in, y)
        out = rt.buf("gattn.out", n, self.o_dim)
        self.mix(ctx, y, cache, out, parts=parts)
        return project(rt, "attn.proj", out, self.w_o, ctx)
