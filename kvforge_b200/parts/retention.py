"""Retention: linear attention with one fixed decay a head, no softmax and no denominator (with silu on the projections
and one norm over all heads it is what is called lightning attention).

Per layer ``q = W_q x``, ``k = W_k x`` (``H`` heads of ``head_dim``), ``v = W_v x`` (``H`` heads of ``v_head_dim``),
``g = W_g x``.  The first ``rotary_dim`` dims of every query and key head turn with the position; the keys are then
multiplied by ``head_dim^(-1/2)``.  Per head a matrix state ``S [head_dim, v_head_dim]`` is carried from token to
token, ``S_t = a_h S_(t-1) + k_t v_t^T``, and read out as ``o_t = S_t^T q_t``.  Every head's ``o`` is divided by its
root mean square (or all heads together are normed with a weight), the heads are multiplied by ``silu(g)`` (or the
logistic function of ``g``) and projected back.  The state is the mixer's state slot
per request: 32-bit floats, zero for a new request; the mixer keeps no pages.
"""

from __future__ import annotations

import torch

from .. import ops
from .base import CacheNeed, Mixer, PartSpec, WeightDecl, build_part, register_mixer
from .gated_attention import stack_rows
from .projection import project


@register_mixer("retention")
class Retention(Mixer):
    """params: ``hidden_size``, ``num_heads``, ``head_dim``, ``v_head_dim``, ``decay`` (a list of ``num_heads`` numbers),
    ``eps`` (of the heads' norm); optional ``position`` (a rotary ``PartSpec`` or ``None``), ``key_scale`` (default
    ``head_dim^(-1/2)``), ``gate`` (``"silu"``, ``"sigmoid"`` or ``None``; default ``"silu"``), ``activation`` (``"silu"``: q, k and v
    pass it right after their projections) and ``norm`` (``"heads"``, the default: every head by itself, without a weight;
    ``"joint"``: the concatenated heads together, with the tensor ``norm [H*v_head_dim]``).

    Tensors: ``q [H*head_dim, W]``, ``k [H*head_dim, W]``, ``v [H*v_head_dim, W]``, ``g [H*v_head_dim, W]`` (with a gate),
    ``o [W, H*v_head_dim]``.

    With the joint norm it also has the open form that ``summed_mixers`` takes: ``take_input`` / ``take_output`` hand the input
    and output matrices over, and ``mix`` computes what lies between the two products."""

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        p = params
        self.hidden, self.nh = int(p["hidden_size"]), int(p["num_heads"])
        self.dk, self.dv = int(p["head_dim"]), int(p["v_head_dim"])
        self.decay_values = [float(a) for a in p["decay"]]
        if len(self.decay_values) != self.nh:
            raise ValueError("retention needs one decay per head")
        if not 0 < self.dk <= ops.RETENTION_MAX_KEY_DIM or self.dv <= 0:
            raise ValueError(f"retention takes key heads of at most {ops.RETENTION_MAX_KEY_DIM} numbers")
        self.eps = float(p["eps"])
        self.key_scale = float(p.get("key_scale") or self.dk**-0.5)
        self.gate = p.get("gate", "silu")
        if self.gate not in ("silu", "sigmoid", None):
            raise ValueError("the gate of retention is 'silu', 'sigmoid' or None")
        self.activation = p.get("activation")
        if self.activation not in ("silu", None):
            raise ValueError("the activation of retention's projections is 'silu' or None")
        self.norm = p.get("norm", "heads")
        if self.norm not in ("heads", "joint"):
            raise ValueError("the norm of retention is 'heads' or 'joint'")
        pos = p.get("position")
        if isinstance(pos, dict):
            pos = PartSpec(pos["kind"], pos.get("params", {}))
        self.position_spec: PartSpec | None = pos
        self.position = None

    @classmethod
    def weight_decls(cls, params):
        w, h, dk, dv = (int(params[k]) for k in ("hidden_size", "num_heads", "head_dim", "v_head_dim"))
        out = {"q": WeightDecl((h * dk, w)), "k": WeightDecl((h * dk, w)), "v": WeightDecl((h * dv, w)), "o": WeightDecl((w, h * dv))}
        if params.get("gate", "silu") is not None:
            out["g"] = WeightDecl((h * dv, w))
        if params.get("norm", "heads") == "joint":
            out["norm"] = WeightDecl((h * dv,), kind="vector", init="ones")
        return out

    def cache_need(self) -> CacheNeed:
        return CacheNeed("none")

    def state_shape(self):
        return (self.nh * self.dk * self.dv,)

    def bind(self, weights, rt):
        super().bind(weights, rt)
        mats = [weights["q"], weights["k"], weights["v"]] + ([weights["g"]] if self.gate else [])
        # each projection from a multiple of 8 columns of the product on
        self.w_in, offs = stack_rows(mats)
        self.in_dim = self.w_in.shape[0]
        self.k_off, self.v_off = offs[1], offs[2]
        self.g_off = offs[3] if self.gate else None
        self.norm_w = weights["norm"].contiguous() if self.norm == "joint" else None
        self.w_o = weights["o"].contiguous()
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=rt.device)
        # the chunked form works with logarithms: decays in (0, 1]
        self.log_decay = None
        if all(0.0 < a <= 1.0 for a in self.decay_values):
            self.log_decay = torch.tensor(self.decay_values, dtype=torch.float64).log().to(device=rt.device, dtype=torch.float32)
        if self.position_spec is not None and self.position is None:
            self.position = build_part("position", self.position_spec)
            self.position.bind({}, rt)
        if self.position is not None and self.position.magnitude != 1.0:
            raise ValueError("retention turns pairs without changing their size")
        self.inv_freq = self.position.table() if self.position is not None else None
        self.interleaved = bool(getattr(self.position, "pairs_interleaved", False))

    # ------------------------------------------------------------------ between the two products
    inner_width = property(lambda self: self.nh * self.dv)
    open_form = property(lambda self: self.norm == "joint")

    def take_input(self) -> torch.Tensor:
        w, self.w_in = self.w_in, None
        return w

    def take_output(self) -> torch.Tensor:
        w, self.w_o = self.w_o, None
        return w

    def mix(self, ctx, y: torch.Tensor, cache, out: torch.Tensor, mult: float = 1.0) -> None:
        """``y [N, in_dim]``: the input product's rows; ``out [N, inner_width]`` gets ``mult`` times what the output
        projection multiplies."""
        rt, n = self.rt, y.shape[0]
        if cache is None or cache.state is None:
            raise RuntimeError("retention needs its state slots")
        h, dk, dv = self.nh, self.dk, self.dv
        o = rt.buf("retention.o", n, h * dv, torch.float32)
        scratch = (
            rt.buf("retention.qn", n, h * dk, torch.float32),
            rt.buf("retention.kn", n, h * dk, torch.float32),
            rt.buf("retention.vn", n, h * dv, torch.float32),
        )
        # many tokens of few sequences in bfloat16: chunk by chunk; 32-bit: token by token, the same bits however a sequence is cut
        raw = None
        chunked = rt.dtype == torch.bfloat16 and self.log_decay is not None and ops.chunks_pay(ctx.num_seqs, ctx.max_query_len)
        if chunked and ops.chunks_ok(dk, dv, cache.state):
            raw = rt.buf("retention.raw", n, h * ops.CHUNK_TOKENS, torch.float32)
        ops.retention(
            y, 0, self.k_off, self.v_off, ctx.positions, self.inv_freq, self.interleaved, self.key_scale, self.decay, cache.state, o,
            ctx.query_start_loc, ctx.state_slots, ctx.num_seqs, h, dk, dv, scratch, max_query_len=ctx.max_query_len, activation=self.activation,
            log_decay=self.log_decay, raw=raw,
        )  # fmt: skip
        gate = y[:, self.g_off : self.g_off + h * dv] if self.gate else None
        if self.norm == "joint":
            ops.wide_norm_gate(o, self.norm_w, self.eps, out, gate=gate, activation=self.gate, mult=mult)
        elif mult == 1.0:
            ops.retention_gate(o, gate, self.eps, out, h, dv, self.gate)
        else:
            raise RuntimeError("retention with heads normed one by one is not scaled")

    def forward(self, ctx, x: torch.Tensor, cache):
        rt, n = self.rt, x.shape[0]
        y = rt.buf("retention.in", n, self.in_dim)
        if ops.skinny_ok(x, self.w_in):
            ops.gemm_skinny(x, self.w_in, y)
        else:
            ops.linear(x, self.w_in, y)
        out = rt.buf("retention.out", n, self.inner_width)
        self.mix(ctx, y, cache, out)
        return project(rt, "retention.proj", out, self.w_o, ctx)
