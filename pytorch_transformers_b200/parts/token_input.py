"""Inputs that a layer takes straight from the token ids, beside the stream.

``gated_table``: with ``e`` the token's row of a table that all layers share (this layer's ``dim`` columns, from ``first``),

    x <- x + rmsnorm( W_proj ( gelu_tanh(W_gate x) * e ) ) * gain.

The table belongs to the model (``ModelSpec.token_table_name``) and reaches the part through the step (``ctx.token_table``).
The two products' inner size ``dim`` is padded with zeros to what the weight-streaming kernel takes.
"""
from __future__ import annotations

from typing import Dict

import torch

from .base import BuildContext, ParamDecl, Part, PartSpec, register_part
from .linear import linear

MULTIPLE = 32


@register_part("token_input", "gated_table")
class GatedTableInput(Part):
    graph_safe = True

    def __init__(self, build: BuildContext, spec: PartSpec, hidden: int, dim: int, first: int, eps: float):
        super().__init__(build, spec)
        self.hidden, self.dim, self.first, self.eps = int(hidden), int(dim), int(first), float(eps)
        if self.dim <= 0 or self.first < 0:
            raise ValueError(f"a token input takes a positive number of columns from a column >= 0, got {dim} from {first}")
        self.padded = (self.dim + MULTIPLE - 1) // MULTIPLE * MULTIPLE
        self.p_gate = self.p_proj = self.p_norm = None

    def param_decls(self) -> Dict[str, ParamDecl]:
        return {"gate": ParamDecl((self.dim, self.hidden)), "proj": ParamDecl((self.hidden, self.dim)),
                "norm": ParamDecl((self.hidden,), role="vector", init="one_plus_normal", std=0.1)}

    def bind(self, t: Dict[str, torch.Tensor]) -> None:
        self.p_gate = t["gate"].contiguous()
        self.p_proj = t["proj"].new_zeros(self.hidden, self.padded)
        self.p_proj[:, :self.dim] = t["proj"]
        self.p_norm = t["norm"]

    def forward_stream(self, x, h, ctx, copy_dtype):
        """``x`` the float32 stream, ``h`` its copy in the model dtype: (the new stream, its copy)."""
        k = self.build.kernels
        z = linear(k, h, self.p_gate, wide_out=True)
        g = k.token_gate(z, ctx.dev["tokens"], ctx.token_table, self.first, self.dim, self.padded, ctx.status)
        return k.norm_add(x, linear(k, g, self.p_proj, wide_out=True), self.p_norm, self.eps, copy_dtype)
