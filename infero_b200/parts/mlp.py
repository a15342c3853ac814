"""SwiGLU feed-forward."""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import kernels as K
from ..config.spec import FeedForwardSpec
from .base import FeedForward, TensorDecl
from .linear import Linear


class SwiGluMlp(FeedForward):
    """delta = down(silu(gate(h)) * up(h)) (crates/model/src/lib.rs:7391-7451, :7506-7531;
    crates/kernels/src/cu/ops.cu:111-133).  gate and up are stacked into one [2*ff, d]
    matrix at bind time, rows alternating gate_j, up_j, so that one product yields each pair
    side by side: the tensor-core kernel applies the activation in its epilogue, and where it
    cannot (32-bit path, a product cut into several splits) the SwiGLU kernel takes the same
    alternating layout.  Where the tensors live under the block's prefix is data of the spec
    (``FeedForwardSpec.names``): separate gate and up, or one stored [gate; up] tensor.  ``bias``: every projection has
    one (leaf name + ``.b``), added in the products' epilogues or by the kernel that adds up partial sums."""

    def __init__(self, spec: FeedForwardSpec, prefix: str):
        self.spec = spec
        self.prefix = prefix
        self.gate_up: Linear = None
        self.down: Linear = None
        self.names = spec.tensor_names()
        self.stored_stacked = "gate_up" in self.names    # the checkpoint holds one [gate; up] tensor

    def _n(self, role: str) -> str:
        return f"{self.prefix}.{self.names[role]}{self.spec.weight_suffix}"

    def _b(self, role: str) -> str:
        return f"{self.prefix}.{self.names[role]}.b"

    def declare(self) -> List[TensorDecl]:
        d, ff = self.spec.hidden, self.spec.intermediate
        biases = [TensorDecl(self._b(r), (n,), role="bias") for r, n in (("gate", ff), ("up", ff), ("down", d))] if self.spec.bias else []
        if self.stored_stacked:
            if biases:
                raise ValueError("biases come with separate gate and up tensors")
            return [TensorDecl(self._n("gate_up"), (2 * ff, d)), TensorDecl(self._n("down"), (d, ff))]
        return [TensorDecl(self._n("gate"), (ff, d)), TensorDecl(self._n("up"), (ff, d)),
                TensorDecl(self._n("down"), (d, ff))] + biases

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        if self.stored_stacked:
            g, u = tensors[self._n("gate_up")].chunk(2, dim=0)
        else:
            g, u = tensors[self._n("gate")], tensors[self._n("up")]
        if g.dtype != u.dtype:
            g, u = g.float(), u.float()
        gu_bias = down_bias = None
        if self.spec.bias:
            gu_bias = torch.stack([tensors[self._b("gate")].float(), tensors[self._b("up")].float()], dim=1).reshape(-1).contiguous()
            down_bias = tensors[self._b("down")].float().contiguous()
        self.gate_up = Linear(torch.stack([g, u], dim=1).reshape(2 * g.shape[0], g.shape[1]), gu_bias,
                              f"{self.prefix}.gate_up")
        self.down = Linear(tensors[self._n("down")], down_bias, self._n("down"))

    def forward(self, ctx, h):
        T = h.shape[0]
        act = torch.empty((T, self.spec.intermediate), dtype=h.dtype, device=h.device)
        if not self.gate_up.forward_swiglu(h, act):
            if self.spec.bias:
                from ..kernels import layer_ops as L
                L.glu_act(self.gate_up.forward(h, defer=True, out_dtype=torch.float32), act)
                return self.down.forward(act, defer=True, residual=True)
            K.swiglu(self.gate_up.forward(h, defer=True), act)
        return self.down.forward(act, defer=True, residual=True)


class GluMlp(SwiGluMlp):
    """delta = down(glu(gate(h), up(h))) with one of the gated activations of the kernels (``activation`` "swiglu" or
    "glu_clamped" with ``limit`` and ``act_alpha``); the stacked layout of ``SwiGluMlp``.  The plain SwiGLU case keeps
    the base class's fused epilogue; the others run the product and then the activation kernel."""

    def forward(self, ctx, h):
        s = self.spec
        if s.activation == "swiglu":
            return super().forward(ctx, h)
        if s.bias:
            raise ValueError("the clamped activation comes without biases")
        from ..kernels import layer_ops as L, tc_gemm
        act = torch.empty((h.shape[0], s.intermediate), dtype=h.dtype, device=h.device)
        # many rows in bf16: the activation in the product's epilogue; else the product (as partial sums where it is cut)
        # and the activation kernel
        if not (h.dtype == torch.bfloat16 and self.gate_up.weight.dtype == torch.bfloat16
                and tc_gemm.gemm_act(h, self.gate_up.weight, act, s.activation, s.limit, s.act_alpha)):
            L.glu_act(self.gate_up.forward(h, defer=True), act, (s.activation, s.limit, s.act_alpha))
        return self.down.forward(act, defer=True, residual=True)


class Relu2Mlp(FeedForward):
    """delta = down(relu(up(h))^2)."""

    def __init__(self, spec: FeedForwardSpec, prefix: str):
        self.spec, self.prefix = spec, prefix
        self.names = spec.tensor_names()
        self.up: Linear = None
        self.down: Linear = None

    def _n(self, role: str) -> str:
        return f"{self.prefix}.{self.names[role]}{self.spec.weight_suffix}"

    def declare(self) -> List[TensorDecl]:
        d, ff = self.spec.hidden, self.spec.intermediate
        return [TensorDecl(self._n("up"), (ff, d)), TensorDecl(self._n("down"), (d, ff))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.up = Linear(tensors[self._n("up")], None, self._n("up"))
        self.down = Linear(tensors[self._n("down")], None, self._n("down"))

    def forward(self, ctx, h):
        from ..kernels import layer_ops as L, tc_gemm
        act = torch.empty((h.shape[0], self.spec.intermediate), dtype=h.dtype, device=h.device)
        if not (h.dtype == torch.bfloat16 and self.up.weight.dtype == torch.bfloat16
                and tc_gemm.gemm_act(h, self.up.weight, act, "relu2")):
            L.relu2(self.up.forward(h, defer=True), act)
        return self.down.forward(act, defer=True, residual=True)
