"""A selective state space as a mixer (the recurrence of Mamba-2): a matrix state per head instead of pages of keys.

One projection of the input holds, in this order, a gate ``z [inner]``, ``x [inner]``, ``B [G*N]``, ``C [G*N]`` and a step-size
logit per head (``inner = heads * v_head_dim``).  ``x``, ``B`` and ``C`` pass a short causal convolution over time per channel
(with a bias) and SiLU.  With ``d = softplus(dt + dt_bias)``, per head (head ``h`` takes group ``h // (heads / G)``)::

    S <- exp(-exp(A_log) d) S + d B x^T        y = S^T C + D x        (S [N, v_head_dim])

The read-out is multiplied by ``silu(z)`` first and RMS-normed after, in ``norm_groups`` equal parts, with a weight as wide as
``inner``; then the output projection.  What the recurrence reads besides the convolution's result is float in both storage
types: step sizes, decays, the state.  A request's state is one row of floats: the last ``conv - 1`` inputs of the
convolution, then ``S``.
"""

from __future__ import annotations

import torch

from .. import ops
from .base import Mixer, WeightDecl, register_mixer
from .gated_attention import stack_rows
from .projection import project


@register_mixer("state_space")
class StateSpace(Mixer):
    """params: ``hidden_size``, ``num_heads``, ``v_head_dim``, ``state_dim`` (N), ``groups`` (G), ``conv`` (taps), ``norm_groups``,
    ``eps``.  Tensors: ``in``, ``conv``, ``conv.b``, ``dt_bias``, ``A_log``, ``D``, ``norm``, ``o``."""

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        p = params
        self.hidden, self.H, self.dv = int(p["hidden_size"]), int(p["num_heads"]), int(p["v_head_dim"])
        self.N, self.G, self.taps = int(p["state_dim"]), int(p["groups"]), int(p["conv"])
        self.norm_groups, self.eps = int(p["norm_groups"]), float(p["eps"])
        self.inner = self.H * self.dv
        if self.G <= 0 or self.H % self.G:
            raise ValueError("num_heads must be a multiple of groups")
        if self.norm_groups <= 0 or self.inner % self.norm_groups:
            raise ValueError("norm_groups must divide num_heads * v_head_dim")
        if not 0 < self.N <= ops.STATE_SPACE_MAX_STATE or self.taps < 1:
            raise ValueError(f"state_dim must be between 1 and {ops.STATE_SPACE_MAX_STATE}, conv at least 1 tap")
        self.c_conv = self.inner + 2 * self.G * self.N
        self.conv_floats = (self.taps - 1) * self.c_conv
        self.state_floats = self.conv_floats + self.H * self.N * self.dv

    @classmethod
    def weight_decls(cls, params):
        p = params
        w, H, dv, N, G, taps = (int(p[k]) for k in ("hidden_size", "num_heads", "v_head_dim", "state_dim", "groups", "conv"))
        inner = H * dv
        return {
            "in": WeightDecl((2 * inner + 2 * G * N + H, w)),
            "conv": WeightDecl((inner + 2 * G * N, taps), kind="vector", init="conv"),
            "conv.b": WeightDecl((inner + 2 * G * N,), kind="vector", init="zeros"),
            "dt_bias": WeightDecl((H,), kind="vector", init="small"),
            "A_log": WeightDecl((H,), kind="vector", init="small"),
            "D": WeightDecl((H,), kind="vector", init="ones"),
            "norm": WeightDecl((inner,), kind="vector", init="ones"),
            "o": WeightDecl((w, inner)),
        }

    def state_shape(self):
        return (self.state_floats,)

    def bind(self, weights, rt):
        super().bind(weights, rt)
        z, xbc, dt = weights["in"].split([self.inner, self.c_conv, self.H], dim=0)
        # each stretch from a multiple of 8 columns of the product on
        self.w_in, (self.z_off, self.x_off, self.dt_off) = stack_rows([z, xbc, dt])
        self.in_dim = self.w_in.shape[0]
        self.w_o = weights["o"].contiguous()
        self.w_conv, self.b_conv = weights["conv"].t().contiguous(), weights["conv.b"].contiguous()
        self.dt_bias, self.a_log, self.skip, self.norm_w = (weights[k].contiguous() for k in ("dt_bias", "A_log", "D", "norm"))

    def forward(self, ctx, x: torch.Tensor, cache):
        rt, n = self.rt, x.shape[0]
        if cache is None or cache.state is None:
            raise RuntimeError("state_space needs a state slot per request")
        H, dv, gn = self.H, self.dv, self.G * self.N
        y = rt.buf("ssm.in", n, self.in_dim)
        if ops.skinny_ok(x, self.w_in):
            ops.gemm_skinny(x, self.w_in, y)
        else:
            ops.linear(x, self.w_in, y)
        xbc = rt.buf("ssm.xbc", n, self.c_conv)
        ops.causal_conv(
            y[:, self.x_off : self.x_off + self.c_conv], self.w_conv, cache.state[:, : self.conv_floats], ctx.query_start_loc, ctx.state_slots,
            ctx.num_seqs, xbc, activation="silu", max_query_len=ctx.max_query_len, bias=self.b_conv,
        )  # fmt: skip
        f32 = torch.float32
        read = rt.buf("ssm.read", n, self.inner, f32)
        scratch = (rt.buf("ssm.decay", n, H, f32), rt.buf("ssm.cn", n, gn, f32), rt.buf("ssm.bn", n, gn, f32), rt.buf("ssm.vn", n, self.inner, f32))
        # many tokens of few sequences in bfloat16: chunk by chunk; 32-bit: token by token, the same bits however a sequence is cut
        state, raw = cache.state[:, self.conv_floats :], None
        if rt.dtype == torch.bfloat16 and ops.chunks_pay(ctx.num_seqs, ctx.max_query_len) and ops.chunks_ok(self.N, dv, state):
            raw = rt.buf("ssm.raw", n, self.G * ops.CHUNK_TOKENS, f32)
        ops.state_space(
            xbc, y[:, self.dt_off : self.dt_off + H], self.dt_bias, self.a_log, state, read, ctx.query_start_loc,
            ctx.state_slots, ctx.num_seqs, H, self.G, self.N, dv, scratch, max_query_len=ctx.max_query_len, raw=raw,
        )  # fmt: skip
        out = rt.buf("ssm.out", n, self.inner)
        ops.wide_norm_gate(
            read, self.norm_w, self.eps, out, self.norm_groups, gate=y[:, self.z_off : self.z_off + self.inner], activation="silu", gate_first=True,
            skip=self.skip, skip_x=xbc[:, : self.inner],
        )  # fmt: skip
        return project(rt, "ssm.proj", out, self.w_o, ctx)
