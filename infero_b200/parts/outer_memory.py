"""Recurrences whose state is a matrix per head that every token updates with an outer product."""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..config.spec import MixerSpec
from ..kernels import layer_ops as L
from .base import Mixer, StateSpec, TensorDecl
from .linear import Linear


def single_tokens(ctx) -> bool:
    """Does every request of the step bring one token?"""
    longest = int(getattr(ctx, "max_q_len", 0) or 0)
    return longest == 1 if longest else ctx.n_tokens == ctx.n_entries


class _OuterMemory(Mixer):
    """What the two rules share: a stacked input product in 32-bit, a state vector in the request's slot, and the three
    stages (``input_rows``, ``core``, ``output_weight``) that let the mixer run as a branch of another."""

    RULE = ""

    def __init__(self, spec: MixerSpec, prefix: str):
        self.spec, self.prefix = spec, prefix
        self.H, self.K, self.V = int(spec.num_heads), int(spec.head_dim), int(spec.v_dim)
        if min(self.H, self.K, self.V) <= 0:
            raise ValueError("a memory needs heads, head_dim and value_dim")
        if self.K > 512:
            raise ValueError(f"keys of {self.K}, at most 512")
        self.names = spec.tensor_names()
        self.inp: Linear = None
        self.out: Linear = None

    def _n(self, role: str, matrix: bool = True) -> str:
        return f"{self.prefix}.{self.names[role]}" + (self.spec.weight_suffix if matrix else "")

    def _stack(self) -> List[Tuple[str, int]]:
        """Roles and rows of the input product, in column order."""
        raise NotImplementedError

    def _offsets(self) -> Dict[str, int]:
        at, out = 0, {}
        for role, n in self._stack():
            out[role] = at
            at += n
        self.n_rows = at
        return out

    def _bind_product(self, tensors, bias=None) -> None:
        ws = [tensors[self._n(r)] for r, _ in self._stack()]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.float() for w in ws]
        self._rows, self._bias = torch.cat(ws, dim=0).contiguous(), bias
        self.inp = Linear(self._rows, bias, f"{self.prefix}.{self.RULE}")
        self._out_w = tensors[self._n("o")]
        self.out = Linear(self._out_w, None, self._n("o"))

    def input_rows(self):
        return self._rows, self._bias

    def output_weight(self) -> torch.Tensor:
        return self._out_w

    @property
    def out_width(self) -> int:
        return self.H * self.V

    def forward(self, ctx, h, slot):
        proj = self.inp.forward(h, out_dtype=torch.float32)
        act = torch.empty((h.shape[0], self.H * self.V), dtype=h.dtype, device=h.device)
        self.core(ctx, proj, 0, slot, act)
        return self.out.forward(act, defer=True, residual=True, out_dtype=torch.float32)


class DeltaMemory(_OuterMemory):
    """The gated delta rule.  One input product gives [q | k | v | gate | step | decay]; q and k have ``num_kv_heads`` heads
    of ``head_dim``, v and the gate ``num_heads`` of ``value_dim``.  ``memory_prepare`` (convolution, silu, unit vectors, gates) ->
    ``delta_scan`` -> ``memory_finish`` (RMS norm with a weight shared by the heads, silu gate) -> output product.  The
    request's state: the convolution's last taps - 1 inputs, then S."""

    RULE = "delta"

    def __init__(self, spec: MixerSpec, prefix: str):
        super().__init__(spec, prefix)
        self.G, self.taps = int(spec.num_kv_heads) or self.H, int(spec.conv_taps)
        if self.H % self.G:
            raise ValueError(f"{self.H} heads are not a multiple of {self.G} kv heads")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"{self.taps} taps outside 1..16")
        self.CH = 2 * self.G * self.K + self.H * self.V
        self.off = self._offsets()
        self.s_off = L.memory_tail_floats(self.taps, self.CH)

    def _stack(self):
        return [("q", self.G * self.K), ("k", self.G * self.K), ("v", self.H * self.V), ("gate", self.H * self.V),
                ("step", self.H), ("decay", self.H)]

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((L.memory_state_floats("delta", self.H, self.K, self.V, self.taps, self.CH),), torch.float32)

    def declare(self) -> List[TensorDecl]:
        d = self.spec.hidden
        out = [TensorDecl(self._n(r), (n, d)) for r, n in self._stack()]
        out += [TensorDecl(self._n(r + "_conv", False), (n, self.taps), role="bias", init="conv") for r, n in self._stack()[:3]]
        return out + [TensorDecl(self._n("dt_bias", False), (self.H,), role="bias"), TensorDecl(self._n("a_log", False), (self.H,), role="bias"),
                      TensorDecl(self._n("out_norm", False), (self.V,), role="norm", init="ones"),
                      TensorDecl(self._n("o"), (d, self.H * self.V))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        f32 = lambda r: tensors[self._n(r, False)].float().contiguous()          # noqa: E731
        self._bind_product(tensors)
        self.conv_w = torch.cat([f32(r + "_conv") for r in ("q", "k", "v")], dim=0).t().contiguous()      # [taps, channels]
        self.dt_bias, self.a_log, self.norm_w = f32("dt_bias"), f32("a_log"), f32("out_norm")

    def core(self, ctx, proj: torch.Tensor, off: int, slot, out: torch.Tensor, scale: float = 1.0) -> None:
        H, G, K, V, o = self.H, self.G, self.K, self.V, self.off
        state = ctx.state(slot.cache)
        single = single_tokens(ctx)
        batch = (ctx.entry_q_start, ctx.entry_q_len, ctx.entry_slot, ctx.n_entries)
        u, table = L.memory_prepare(proj, off, off + o["decay"], off + o["step"], self.conv_w, self.a_log, self.dt_bias, state, ctx.tok_entry,
                                    *batch, G, H, K, V, single)
        y = L.delta_scan(u, table, state, self.s_off, *batch, H, G, K, V, single)
        L.memory_finish(y, None, proj[:, off + o["gate"]:off + o["gate"] + H * V], "silu", self.norm_w, float(self.spec.norm_eps),
                        out, H, V, scale)


class GatedMemory(_OuterMemory):
    """The matrix memory of an mLSTM (exponential gates, a normaliser and a running maximum).  One input product gives
    [q | k | v | gate | input | forget], every head with its own q and k; ``gated_scan`` -> ``memory_finish`` (division by
    the normaliser, root mean square per head, a weight over all heads, sigmoid gate) -> output product.  The request's
    state: S with the normaliser as one more column, and the maximum."""

    RULE = "gated"

    def __init__(self, spec: MixerSpec, prefix: str):
        super().__init__(spec, prefix)
        if not spec.gate_cap > 0:
            raise ValueError("a gated memory needs gate_cap")
        self.off = self._offsets()

    def _stack(self):
        return [("q", self.H * self.K), ("k", self.H * self.K), ("v", self.H * self.V), ("gate", self.H * self.V),
                ("input", self.H), ("forget", self.H)]

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((L.memory_state_floats("gated", self.H, self.K, self.V),), torch.float32)

    def declare(self) -> List[TensorDecl]:
        d = self.spec.hidden
        return [TensorDecl(self._n(r), (n, d)) for r, n in self._stack()] + [
            TensorDecl(self._n("input_bias", False), (self.H,), role="bias"), TensorDecl(self._n("forget_bias", False), (self.H,), role="bias"),
            TensorDecl(self._n("out_norm", False), (self.H * self.V,), role="norm", init="ones"),
            TensorDecl(self._n("o"), (d, self.H * self.V))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        f32 = lambda r: tensors[self._n(r, False)].float().contiguous()          # noqa: E731
        i_b, f_b = f32("input_bias"), f32("forget_bias")
        zeros = torch.zeros(self.n_rows - 2 * self.H, dtype=torch.float32, device=i_b.device)
        self._bind_product(tensors, torch.cat([zeros, i_b, f_b]).contiguous())
        self.norm_w = f32("out_norm")

    def core(self, ctx, proj: torch.Tensor, off: int, slot, out: torch.Tensor, scale: float = 1.0) -> None:
        H, K, V, o = self.H, self.K, self.V, self.off
        y, den = L.gated_scan(proj, off + o["q"], off + o["k"], off + o["v"], off + o["input"], off + o["forget"], float(self.spec.gate_cap),
                              ctx.state(slot.cache), 0, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_slot, ctx.n_entries, H, K, V,
                              single_tokens(ctx))
        L.memory_finish(y, den, proj[:, off + o["gate"]:off + o["gate"] + H * V], "sigmoid", self.norm_w, float(self.spec.norm_eps),
                        out, H, V, scale)


class _ChannelDecayed(_OuterMemory):
    """Memories whose every key channel decays on its own.  The decays (and a gate, where the rule has one of that kind) are
    products through a narrow middle, W_up (W_down h): the rows of W_down ride on the stacked input product and ``low_rank``
    does the rest in 32-bit.  How wide a middle is only the stored tensors say (``spec.low_rank`` where weights are made)."""

    NARROW: Tuple[str, ...] = ()             # roles of the W_down

    def __init__(self, spec: MixerSpec, prefix: str):
        super().__init__(spec, prefix)
        self.ranks = {r: int(spec.low_rank) for r in self.NARROW}
        if min(self.ranks.values()) <= 0:
            raise ValueError("a product through a narrow middle needs low_rank")
        self.off = self._offsets()

    def _declare_rows(self) -> List[TensorDecl]:
        d = self.spec.hidden
        return [TensorDecl(self._n(r), (n, d), free_axes=(0,) if r in self.NARROW else ()) for r, n in self._stack()]

    def _bind_rows(self, tensors) -> None:
        """The stacked product, its width rounded up to whole vectors of four."""
        self.ranks = {r: tensors[self._n(r)].shape[0] for r in self.NARROW}
        self.off = self._offsets()
        self._bind_product(tensors)
        pad = -self.n_rows % 4
        if pad:
            self._rows = torch.cat([self._rows, torch.zeros((pad, self._rows.shape[1]), dtype=self._rows.dtype, device=self._rows.device)])
            self.inp = Linear(self._rows, None, self.inp.name)

    def _up(self, tensors, role: str, down: str) -> torch.Tensor:
        w = tensors[self._n(role)].contiguous()
        if w.shape[1] != self.ranks[down]:
            raise ValueError(f"{self._n(role)} takes {w.shape[1]} numbers, {self._n(down)} gives {self.ranks[down]}")
        return w

    def _narrow(self, proj: torch.Tensor, off: int, role: str) -> torch.Tensor:
        at = off + self.off[role]
        return proj[:, at:at + self.ranks[role]]


class ChannelDeltaMemory(_ChannelDecayed):
    """The gated delta rule with a decay per key channel.  One input product gives [q | k | v | decay's middle | gate's middle |
    step]; ``low_rank`` makes the decays exp(-exp(A_log) softplus(W_a2 (W_a1 h) + dt_bias)) and the gate, then
    ``channel_prepare`` (convolution, silu, unit vectors, what the scan reads of every group of four tokens) -> ``channel_scan``
    -> ``memory_finish`` (RMS norm with a weight shared by the heads, sigmoid gate) -> output product.  The request's state: the
    convolution's last taps - 1 inputs, then S."""

    RULE = "channel_delta"
    NARROW = ("decay_down", "gate_down")

    def __init__(self, spec: MixerSpec, prefix: str):
        self.G, self.taps = int(spec.num_kv_heads) or int(spec.num_heads), int(spec.conv_taps)
        super().__init__(spec, prefix)
        if self.H % self.G:
            raise ValueError(f"{self.H} heads are not a multiple of {self.G} kv heads")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"{self.taps} taps outside 1..16")
        self.CH = 2 * self.G * self.K + self.H * self.V
        self.s_off = L.memory_tail_floats(self.taps, self.CH)

    def _stack(self):
        return [("q", self.G * self.K), ("k", self.G * self.K), ("v", self.H * self.V), ("decay_down", self.ranks["decay_down"]),
                ("gate_down", self.ranks["gate_down"]), ("step", self.H)]

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((L.memory_state_floats("delta", self.H, self.K, self.V, self.taps, self.CH),), torch.float32)

    def declare(self) -> List[TensorDecl]:
        d, r = self.spec.hidden, self.ranks
        out = self._declare_rows()
        out += [TensorDecl(self._n(n + "_conv", False), (w, self.taps), role="bias", init="conv") for n, w in self._stack()[:3]]
        return out + [TensorDecl(self._n("decay_up"), (self.H * self.K, r["decay_down"]), free_axes=(1,)),
                      TensorDecl(self._n("gate_up"), (self.H * self.V, r["gate_down"]), free_axes=(1,)),
                      TensorDecl(self._n("dt_bias", False), (self.H * self.K,), role="bias"), TensorDecl(self._n("a_log", False), (self.H,), role="bias"),
                      TensorDecl(self._n("out_norm", False), (self.V,), role="norm", init="ones"),
                      TensorDecl(self._n("o"), (d, self.H * self.V))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        f32 = lambda r: tensors[self._n(r, False)].float().contiguous()          # noqa: E731
        self._bind_rows(tensors)
        self.decay_up, self.gate_up = self._up(tensors, "decay_up", "decay_down"), self._up(tensors, "gate_up", "gate_down")
        self.conv_w = torch.cat([f32(r + "_conv") for r in ("q", "k", "v")], dim=0).t().contiguous()      # [taps, channels]
        self.dt_bias, self.a_log, self.norm_w = f32("dt_bias"), f32("a_log"), f32("out_norm")

    def core(self, ctx, proj: torch.Tensor, off: int, slot, out: torch.Tensor, scale: float = 1.0) -> None:
        H, G, K, V = self.H, self.G, self.K, self.V
        state, single = ctx.state(slot.cache), single_tokens(ctx)
        decay, gate = L.low_rank(self._narrow(proj, off, "decay_down"), self.decay_up, "decay", self.dt_bias, self.a_log,
                                 beside=(self._narrow(proj, off, "gate_down"), self.gate_up))
        batch = (ctx.entry_q_start, ctx.entry_q_len, ctx.entry_slot, ctx.n_entries)
        v, rec = L.channel_prepare(proj, off, off + self.off["step"], self.conv_w, decay, state, ctx.tok_entry, *batch, G, H, K, V, single)
        y = L.channel_scan(v, rec, state, self.s_off, *batch, H, K, V, single)
        L.memory_finish(y, None, gate, "sigmoid", self.norm_w, float(self.spec.norm_eps), out, H, V, scale)


class DecayedMemory(_ChannelDecayed):
    """Gated linear attention: S <- diag(a) S + k v^T, o = S^T q, with decays a = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau) per key
    channel and every head its own q and k.  One input product gives [q | k | v | gate | decay's middle]; ``decayed_records`` (decays beside k and q)
    -> ``decayed_scan`` -> ``memory_finish`` (RMS norm with a weight shared by the heads, silu gate) -> output product.  The
    request's state: S."""

    RULE = "decayed"
    NARROW = ("decay_down",)

    def __init__(self, spec: MixerSpec, prefix: str):
        super().__init__(spec, prefix)
        if not spec.decay_tau > 0:
            raise ValueError("gated linear attention needs decay_tau")

    def _stack(self):
        return [("q", self.H * self.K), ("k", self.H * self.K), ("v", self.H * self.V), ("gate", self.H * self.V),
                ("decay_down", self.ranks["decay_down"])]

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((L.memory_state_floats("delta", self.H, self.K, self.V),), torch.float32)

    def declare(self) -> List[TensorDecl]:
        return self._declare_rows() + [
            TensorDecl(self._n("decay_up"), (self.H * self.K, self.ranks["decay_down"]), free_axes=(1,)),
            TensorDecl(self._n("decay_bias", False), (self.H * self.K,), role="bias"),
            TensorDecl(self._n("out_norm", False), (self.V,), role="norm", init="ones"),
            TensorDecl(self._n("o"), (self.spec.hidden, self.H * self.V))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        f32 = lambda r: tensors[self._n(r, False)].float().contiguous()          # noqa: E731
        self._bind_rows(tensors)
        self.decay_up = self._up(tensors, "decay_up", "decay_down")
        self.decay_bias, self.norm_w = f32("decay_bias"), f32("out_norm")

    def core(self, ctx, proj: torch.Tensor, off: int, slot, out: torch.Tensor, scale: float = 1.0) -> None:
        H, K, V, o = self.H, self.K, self.V, self.off
        rec = L.decayed_records(self._narrow(proj, off, "decay_down"), self.decay_up, self.decay_bias, float(self.spec.decay_tau), proj,
                                off + o["q"], off + o["k"], H, K)
        y = L.decayed_scan(proj[:, off + o["v"]:off + o["v"] + H * V], rec, ctx.state(slot.cache), 0, ctx.entry_q_start, ctx.entry_q_len,
                           ctx.entry_slot, ctx.n_entries, H, K, V, single_tokens(ctx))
        L.memory_finish(y, None, proj[:, off + o["gate"]:off + o["gate"] + H * V], "silu", self.norm_w, float(self.spec.norm_eps), out,
                        H, V, scale)
