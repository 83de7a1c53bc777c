"""Mixers side by side: every branch reads the same input.  ``parallel_mixers``: each result is RMS-normed over the
model width with a weight of its own (a plain weight, not one-plus), and the mixer's result is the
mean of the normed results.  ``summed_mixers``: the mixer's result is the sum of the branches' results, each times a
constant.

The branches are ordinary mixers.  At most one of them may keep pages of keys and values (the
block's cache group is that branch's); their per-request states lie side by side in one row of
floats, and each branch is handed its columns.
"""

from __future__ import annotations

import torch

from .. import ops
from .base import CacheNeed, Mixer, PartSpec, WeightDecl, build_part, register_mixer
from .gated_attention import stack_rows
from .projection import project


def _spec(v) -> PartSpec:
    return v if isinstance(v, PartSpec) else PartSpec(v["kind"], v.get("params", {}))


def stack_inputs(branches: list) -> tuple[torch.Tensor, list[tuple[int, int]]]:
    """The input matrices of branches in the open form, one below the other, each from a multiple of 8 rows on, and where each lies."""
    mats = [b.take_input() for b in branches]
    stacked, offs = stack_rows(mats)
    return stacked, [(at, at + m.shape[0]) for at, m in zip(offs, mats)]


def input_product(x: torch.Tensor, w: torch.Tensor, y: torch.Tensor) -> None:
    if ops.skinny_ok(x, w):
        ops.gemm_skinny(x, w, y)
    else:
        ops.linear(x, w, y)


class _SideBySide(Mixer):
    """params: ``hidden_size`` and ``branches``, a list whose entries begin with ``(name, PartSpec)``; branch ``name`` has its
    tensors under ``<prefix><name>.``."""

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden = int(params["hidden_size"])
        self.names = [entry[0] for entry in params["branches"]]
        if not 0 < len(self.names) <= ops.MAX_BRANCHES:
            raise ValueError(f"between 1 and {ops.MAX_BRANCHES} branches")
        self.branches: list[Mixer] = [build_part("mixer", _spec(entry[1]), f"{prefix}{entry[0]}.") for entry in params["branches"]]
        paged = [b for b in self.branches if b.cache_need().kind != "none"]
        if len(paged) > 1:
            raise ValueError("only one branch of parallel mixers may keep pages of keys and values")
        self._need = paged[0].cache_need() if paged else CacheNeed("none")
        self._state_cols: list[tuple[int, int] | None] = []
        at = 0
        for b in self.branches:
            shape = b.state_shape()
            if shape is None:
                self._state_cols.append(None)
                continue
            if len(shape) != 1:
                raise ValueError("a branch's state must be a flat row of floats")
            self._state_cols.append((at, at + shape[0]))
            at += shape[0]
        self._state_floats = at

    def sub_parts(self):
        return list(self.branches)

    def cache_need(self) -> CacheNeed:
        return self._need

    def state_shape(self):
        return (self._state_floats,) if self._state_floats else None

    def branch_view(self, cache, cols):
        """What a branch is handed of the layer's cache: the pages and its own columns of the state."""
        if cache is not None and cache.state is not None:
            return cache.with_state(*cols) if cols else cache.with_state(0, 0)
        return cache


@register_mixer("parallel_mixers")
class ParallelMixers(_SideBySide):
    """params: ``hidden_size``, ``eps``, ``branches``: a list of ``(name, PartSpec)``; branch
    ``name`` has its tensors under ``<prefix><name>.`` and its norm weight is ``<prefix><name>.out``.

    When every branch has the open form (``open_form``: ``take_input``, ``mix``, ``take_output``, and ``read_input`` where a branch makes more
    of the input than that product), their input matrices are one product.  Where a block lets its parts add into the
    residual stream, the mean joins it in the kernel that makes it."""

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.eps = float(params["eps"])

    @classmethod
    def weight_decls(cls, params):
        h = int(params["hidden_size"])
        return {f"{name}.out": WeightDecl((h,), kind="vector", init="ones") for name, _ in params["branches"]}

    def bind(self, weights, rt):
        super().bind(weights, rt)
        self.out_w = [weights[f"{name}.out"] for name in self.names]
        self.open = len(self.branches) > 1 and all(getattr(b, "open_form", False) for b in self.branches)
        if self.open:
            self.w_in, self.in_cols = stack_inputs(self.branches)
            self.w_out = [b.take_output() for b in self.branches]

    def _open_results(self, ctx, x, cache):
        rt, n = self.rt, x.shape[0]
        for b in self.branches:
            if hasattr(b, "read_input"):
                b.read_input(ctx, x)
        y = rt.buf("parallel.in", n, self.w_in.shape[0])
        input_product(x, self.w_in, y)
        results = []
        for i, (branch, cols, (lo, hi)) in enumerate(zip(self.branches, self._state_cols, self.in_cols)):
            inner = rt.buf(f"parallel.inner{i}", n, branch.inner_width)
            branch.mix(ctx, y[:, lo:hi], self.branch_view(cache, cols), inner)
            results.append(project(rt, f"parallel.proj{i}", inner, self.w_out[i], ctx))
        return results

    def _branch_results(self, ctx, x, cache):
        results = []
        for branch, cols in zip(self.branches, self._state_cols):
            y = branch.forward(ctx, x, self.branch_view(cache, cols))
            t = y.t if isinstance(y, ops.Partials) else y
            if any(t.data_ptr() == (o.t if isinstance(o, ops.Partials) else o).data_ptr() for o in results):
                # two branches of one kind hand back the same persistent buffer: keep this one's result apart
                kept = self.rt.buf(f"parallel.keep{len(results)}", t.numel() // t.shape[-1], t.shape[-1], t.dtype).view(t.shape)
                kept.copy_(t)
                y = ops.Partials(kept) if isinstance(y, ops.Partials) else kept
            results.append(y)
        return results

    def forward(self, ctx, x, cache):
        # a branch's result is normed before it is added anywhere
        (keep, ctx.residual), (row, ctx.slices) = (ctx.residual, None), (getattr(ctx, "slices", None), None)
        try:
            results = self._open_results(ctx, x, cache) if self.open else self._branch_results(ctx, x, cache)
        finally:
            ctx.residual, ctx.slices = keep, row
        if keep is not None and keep.shape[0] >= x.shape[0] and keep.shape[1] == self.hidden:
            ops.branch_norm_mean(results, self.out_w, self.eps, keep[: x.shape[0]], add=True)
            return ops.ADDED
        out = self.rt.buf("parallel.out", x.shape[0], self.hidden)
        ops.branch_norm_mean(results, self.out_w, self.eps, out)
        return out


@register_mixer("summed_mixers")
class SummedMixers(_SideBySide):
    """``sum_b scale_b * branch_b(x)``.  params: ``hidden_size``, ``branches``: a list of ``(name, PartSpec, scale)``.

    The branches must have the open form (``take_input``, ``mix``, ``take_output``): their input matrices become one product
    of ``x``, each branch's constant is applied in the kernel that writes what its output projection multiplies (in
    float, before the one rounding), and the output projections side by side are one product whose sum over the inner
    width is the sum of the branches."""

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.scales = [float(entry[2]) for entry in params["branches"]]
        for b in self.branches:
            if not all(hasattr(b, name) for name in ("take_input", "mix", "take_output", "inner_width")):
                raise ValueError(f"{b.kind} has no open form: it cannot be a branch of summed_mixers")

    def bind(self, weights, rt):
        super().bind(weights, rt)  # the branches are bound already: they hand over their matrices
        self.w_in, self.in_cols = stack_inputs(self.branches)
        self.out_cols, outs, at = [], [], 0
        for b in self.branches:
            w = b.take_output()
            pad = -w.shape[1] % 8  # every branch begins at a multiple of 8 columns
            outs.append(torch.nn.functional.pad(w, (0, pad)) if pad else w)
            self.out_cols.append((at, at + w.shape[1]))
            at += w.shape[1] + pad
        self.w_o = torch.cat(outs, dim=1).contiguous()
        self.padded = any(hi % 8 for _, hi in self.out_cols)

    def forward(self, ctx, x, cache):
        rt, n = self.rt, x.shape[0]
        y = rt.buf("summed.in", n, self.w_in.shape[0])
        input_product(x, self.w_in, y)
        inner = rt.buf("summed.inner", n, self.w_o.shape[1])
        if self.padded:
            inner.zero_()  # columns between the branches meet zero weights, and must be numbers
        for branch, cols, (lo, hi), (a, b), scale in zip(self.branches, self._state_cols, self.in_cols, self.out_cols, self.scales):
            branch.mix(ctx, y[:, lo:hi], self.branch_view(cache, cols), inner[:, a:b], scale)
        return project(rt, "summed.proj", inner, self.w_o, ctx)
