"""A matrix memory with exponential gates as a mixer (the mLSTM of "xLSTM: Extended Long Short-Term Memory", Beck et al.): a
matrix state per head instead of pages of keys.

Per layer ``q = W_q x / sqrt(head_dim)``, ``k = W_k x`` (``H`` heads of ``head_dim``), ``v = W_v x`` (``H`` heads of ``v_head_dim``) and two
gates a head whose logarithms are ``i = c tanh((W_i x + b_i) / c)`` and ``f = logsigmoid(c tanh((W_f x + b_f) / c))``.  With a running maximum
``m`` (zero before the first token)::

    m <- max(f + m, i)
    S <- e^(f + m_before - m) S + e^(i - m) k v^T        n <- e^(f + m_before - m) n + e^(i - m) k
    o = S^T q / (max(|n . q|, e^(-m)) + 1e-6)

The read-out is scaled to unit root mean square head by head; a weight as wide as all heads and ``sigmoid(W_g x)`` multiply it before
the output projection.  Everything from the gates' logits on is 32-bit.  A request's state is one row of
floats: per head ``S`` with ``n`` as one more column (``ops.memory_columns``), then the heads' ``m``; the mixer keeps no pages.
"""

from __future__ import annotations

import torch

from .. import ops
from .base import Mixer, WeightDecl, register_mixer
from .gated_attention import stack_rows
from .projection import project


@register_mixer("matrix_memory")
class MatrixMemory(Mixer):
    """params: ``hidden_size``, ``num_heads``, ``head_dim``, ``v_head_dim``, ``gate_cap`` (c), ``eps`` (of the heads' norm).  Tensors: ``q``, ``k``
    ``[H*head_dim, W]``, ``v``, ``g`` ``[H*v_head_dim, W]``, ``o [W, H*v_head_dim]``, ``norm [H*v_head_dim]``, ``i``, ``f`` ``[H, W]``, ``i.b``, ``f.b`` ``[H]``.

    It has the open form that mixers side by side take (``take_input``, ``mix``, ``take_output``); the gates' logits, which are floats, are a
    product of their own (``read_input``)."""

    open_form = True
    inner_width = property(lambda self: self.H * self.dv)

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        p = params
        self.hidden, self.H, self.dk, self.dv = (int(p[k]) for k in ("hidden_size", "num_heads", "head_dim", "v_head_dim"))
        self.cap, self.eps = float(p["gate_cap"]), float(p["eps"])
        if not 0 < self.dk <= ops.MEMORY_MAX_KEY_DIM or not 0 < self.dv <= ops.MEMORY_MAX_VALUE_DIM or self.H <= 0:
            raise ValueError(f"matrix_memory takes key heads of 1 to {ops.MEMORY_MAX_KEY_DIM} numbers and value heads of 1 to {ops.MEMORY_MAX_VALUE_DIM}")
        if not self.cap > 0:
            raise ValueError("gate_cap must be positive")
        self.dvx = ops.memory_columns(self.dv)
        self.state_floats = self.H * self.dk * self.dvx + self.H

    @classmethod
    def weight_decls(cls, params):
        w, h, dk, dv = (int(params[k]) for k in ("hidden_size", "num_heads", "head_dim", "v_head_dim"))
        return {
            "q": WeightDecl((h * dk, w)), "k": WeightDecl((h * dk, w)), "v": WeightDecl((h * dv, w)), "g": WeightDecl((h * dv, w)),
            "o": WeightDecl((w, h * dv)), "norm": WeightDecl((h * dv,), kind="vector", init="ones"),
            "i": WeightDecl((h, w)), "f": WeightDecl((h, w)),
            "i.b": WeightDecl((h,), kind="vector", init="small"), "f.b": WeightDecl((h,), kind="vector", init="small"),
        }  # fmt: skip

    def state_shape(self):
        return (-(-self.state_floats // 4) * 4,)  # slots begin on 16-byte boundaries

    def bind(self, weights, rt):
        super().bind(weights, rt)
        self.w_in, (_, self.k_off, self.v_off, self.g_off) = stack_rows([weights[n] for n in ("q", "k", "v", "g")])
        self.in_dim = self.w_in.shape[0]
        self.w_gates, (_, self.f_off) = stack_rows([weights["i"], weights["f"]])
        self.i_bias, self.f_bias, self.norm_w = (weights[n].contiguous() for n in ("i.b", "f.b", "norm"))
        self.w_o = weights["o"].contiguous()
        self.logits = None

    def take_input(self) -> torch.Tensor:
        w, self.w_in = self.w_in, None
        return w

    def take_output(self) -> torch.Tensor:
        w, self.w_o = self.w_o, None
        return w

    def read_input(self, ctx, x: torch.Tensor) -> None:
        """The gates' logits of the step, in float: few output rows, so for a few tokens slices of K in parallel, which the
        recurrence's first kernel sums."""
        rt, n, c = self.rt, x.shape[0], self.w_gates.shape[0]
        if ops.skinny_ok(x, self.w_gates):
            slices = ops.skinny_splits(c, self.hidden, n)
            rows = ops.SKINNY_MAX_SPLIT * ops.SKINNY_MAX_M
            self.logits = ops.Partials(rt.buf("memory.gates_part", slices * n, c, torch.float32, cap=rows).view(slices, n, c))
            ops.gemm_skinny(x, self.w_gates, self.logits)
        else:
            self.logits = rt.buf("memory.gates", n, c, torch.float32)
            ops.linear(x, self.w_gates, self.logits)

    def mix(self, ctx, y: torch.Tensor, cache, out: torch.Tensor, mult: float = 1.0) -> None:
        """``y [N, in_dim]``: the input product's rows; ``out [N, inner_width]`` gets what the output projection multiplies."""
        rt, n = self.rt, y.shape[0]
        if cache is None or cache.state is None:
            raise RuntimeError("matrix_memory needs a state slot per request")
        if mult != 1.0:
            raise RuntimeError("matrix_memory does not scale its result")
        H, dk, dv, dvx, f32 = self.H, self.dk, self.dv, self.dvx, torch.float32
        o, floor = rt.buf("memory.o", n, H * dvx, f32), rt.buf("memory.floor", n, H, f32)
        scratch = (
            rt.buf("memory.decay", n, H, f32), rt.buf("memory.inflow", n, H, f32), rt.buf("memory.qn", n, H * dk, f32),
            rt.buf("memory.kn", n, H * dk, f32), rt.buf("memory.vn", n, H * dvx, f32),
        )  # fmt: skip
        # many tokens of few sequences in bfloat16: chunk by chunk; 32-bit: token by token, the same bits however a sequence is cut
        state, raw = cache.state[:, : self.state_floats], None
        if rt.dtype == torch.bfloat16 and ops.chunks_pay(ctx.num_seqs, ctx.max_query_len) and ops.chunks_ok(dk, dvx, state):
            raw = rt.buf("memory.raw", n, H * ops.CHUNK_TOKENS, f32)
        ops.matrix_memory(
            y, 0, self.k_off, self.v_off, dk**-0.5, self.logits, self.f_off, self.i_bias, self.f_bias, self.cap, state, o, floor,
            ctx.query_start_loc, ctx.state_slots, ctx.num_seqs, H, dk, dv, scratch, max_query_len=ctx.max_query_len, raw=raw,
        )  # fmt: skip
        ops.memory_read(o, floor, self.norm_w, self.eps, out, H, dv, gate=y[:, self.g_off : self.g_off + H * dv])

    def forward(self, ctx, x: torch.Tensor, cache):
        rt, n = self.rt, x.shape[0]
        self.read_input(ctx, x)
        y = rt.buf("memory.in", n, self.in_dim)
        if ops.skinny_ok(x, self.w_in):
            ops.gemm_skinny(x, self.w_in, y)
        else:
            ops.linear(x, self.w_in, y)
        out = rt.buf("memory.out", n, self.inner_width)
        self.mix(ctx, y, cache, out)
        return project(rt, "memory.proj", out, self.w_o, ctx)
