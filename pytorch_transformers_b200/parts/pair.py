"""A mixer made of two: both children read the pair's input ``h`` and the result is ``left_scale * left(h) + right_scale * right(h)``.

Each child is a mixer that can run in two halves around its own projections (the *projected* protocol):

* ``in_weight()``: its input projections stacked into one matrix [rows, hidden];
* ``forward_projected(proj, ctx, entry, out, out_scale)``: from its rows of the projection (a view whose rows
  lie wider apart) to its heads' results times ``out_scale``, written into ``out`` (a view of columns);
* ``out_weight()``: its output projection [hidden, columns of ``out``].

The pair then does one product for all input projections of both children, lets each child work on its
columns, and one product over the concatenated heads with the output matrices side by side: the
weighted sum of the two mixers is that product's own sum over k (the scales go into the heads' values
in float32, before they are rounded for the product). At most one child may keep pages and at most
one a per-sequence state: both use the pair's one cache entry.
"""
from __future__ import annotations

import torch

from .base import BuildContext, ParamDecl, Part, PartSpec, register_part
from .linear import linear


@register_part("mixer", "pair")
class MixerPair(Part):
    graph_safe = True

    def __init__(self, build: BuildContext, spec: PartSpec, left_scale: float = 1.0, right_scale: float = 1.0):
        super().__init__(build, spec)
        self.left, self.right = self.children["left"], self.children["right"]
        self.scales = (float(left_scale), float(right_scale))
        for child in (self.left, self.right):
            for method in ("in_weight", "forward_projected", "out_weight", "out_columns"):
                if not hasattr(child, method):
                    raise ValueError(f"mixer {child.spec.kind!r} cannot be one of a pair: it lacks {method}()")
        if self.left.cache_need() is not None and self.right.cache_need() is not None:
            raise ValueError("both mixers of a pair want pages of the one cache entry")
        if self.left.state_need() is not None and self.right.state_need() is not None:
            raise ValueError("both mixers of a pair want the state of the one cache entry")
        self.p_in = self.p_out = None

    def cache_need(self):
        return self.left.cache_need() or self.right.cache_need()

    def state_need(self):
        return self.left.state_need() or self.right.state_need()

    def planner(self):
        out = []
        for child in (self.left, self.right):
            p = child.planner()
            out += list(p) if isinstance(p, (list, tuple)) else ([p] if p is not None else [])
        return out

    def after_bind(self) -> None:
        """Both children's input projections in one matrix, their output projections side by side."""
        self._join_inputs()
        self.p_out = torch.cat([self.left.out_weight(), self.right.out_weight()], dim=1).contiguous()
        self.left.release_projections()
        self.right.release_projections()

    def _join_inputs(self) -> None:
        rows = [self.left.in_weight(), self.right.in_weight()]
        # the right child's part of the projection starts at a whole 16-byte word (kernels that load 16 bytes at a time)
        self.pad = (-self.left.in_rows()) % 8
        if self.pad:
            rows.insert(1, torch.zeros((self.pad, rows[0].shape[1]), dtype=rows[0].dtype, device=rows[0].device))
        self.rows_l, self.rows_r = rows[0].shape[0], rows[-1].shape[0]
        self.p_in = torch.cat(rows).contiguous()

    def forward(self, x, ctx, entry):
        """float32 [tokens, hidden] (the product's sums, unrounded): a float32 norm or sum follows."""
        k = self.build.kernels
        w_in, w_out = self.p_in, self.p_out
        proj = linear(k, x, w_in)
        rows_l = self.rows_l
        cols_l, cols_r = self.left.out_columns(), self.right.out_columns()
        heads = torch.empty((x.shape[0], cols_l + cols_r), dtype=x.dtype, device=x.device)
        self.left.forward_projected(proj[:, :rows_l], ctx, entry, heads[:, :cols_l], self.scales[0])
        self.right.forward_projected(proj[:, rows_l + self.pad:], ctx, entry, heads[:, cols_l:], self.scales[1])
        return linear(k, heads, w_out, wide_out=True)


@register_part("mixer", "normed_pair")
class NormedMixerPair(MixerPair):
    """A pair whose two results are normed apart before they are summed:

        mult * (rmsnorm(left(h)) * gain_left + rmsnorm(right(h)) * gain_right),

    both norms over the model width. The input projections are one product as in a plain pair; each child has an output
    product of its own, whose float32 sums a block may take as they are (``forward_branches``) to norm and sum them in the
    kernel that forms the stream."""

    def __init__(self, build: BuildContext, spec: PartSpec, hidden: int, eps: float, mult: float = 0.5):
        super().__init__(build, spec)
        self.hidden, self.eps, self.mult = int(hidden), float(eps), float(mult)
        self.p_left_out = self.p_right_out = self.p_left_gain = self.p_right_gain = None

    def param_decls(self):
        return {n: ParamDecl((self.hidden,), role="vector", init="one_plus_normal", std=0.1) for n in ("left_out", "right_out")}

    def bind(self, t) -> None:
        self.p_left_gain, self.p_right_gain = t["left_out"], t["right_out"]

    def after_bind(self) -> None:
        self._join_inputs()
        self.p_left_out, self.p_right_out = self.left.out_weight().contiguous(), self.right.out_weight().contiguous()
        self.left.release_projections()
        self.right.release_projections()

    def forward_branches(self, x, ctx, entry):
        """(left, right): float32 [tokens, hidden] each, before their norms."""
        k = self.build.kernels
        proj = linear(k, x, self.p_in)
        n = x.shape[0]
        left, right = (torch.empty((n, c.out_columns()), dtype=x.dtype, device=x.device) for c in (self.left, self.right))
        self.left.forward_projected(proj[:, :self.rows_l], ctx, entry, left)
        self.right.forward_projected(proj[:, self.rows_l + self.pad:], ctx, entry, right)
        return linear(k, left, self.p_left_out, wide_out=True), linear(k, right, self.p_right_out, wide_out=True)

    def forward(self, x, ctx, entry):
        raise NotImplementedError("a normed pair's branches are normed and summed by the block (forward_branches)")
