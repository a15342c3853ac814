"""A decoder assembled from a ``ModelSpec``: embedding, a schedule of blocks, final norm, head.

Nothing here is specific to one architecture.  The order in which layers run is the
spec's ``schedule`` (a block may appear twice; an entry may read the cache another entry
fills).  The reference's fixed loop is crates/model/src/lib.rs:3899-3949; the final norm
runs only on the rows whose logits are wanted (:4044-4058) and the head product always
returns 32-bit logits (:4075-4214).
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import kernels as K
from ..config.spec import ModelSpec
from ..parts.base import KvCacheSpec, StateSpec, TensorDecl
from ..parts.linear import Linear
from ..registry import part_class


class DecoderModel:
    MODEL = "model"                          # where the states of no layer are found, see ``state_specs``

    def __init__(self, spec: ModelSpec):
        from .. import parts as _parts  # noqa: F401  (registers the built-in parts)
        self.spec = spec
        self.blocks = [part_class("block", b.kind)(b) for b in spec.blocks]
        self.final_norm = part_class("norm", spec.final_norm.kind)(spec.final_norm, spec.final_norm_name)
        self.embed_norm = None
        if spec.embed_norm is not None:
            if spec.embed_norm.kind not in ("rmsnorm", "rmsnorm_centred"):
                raise ValueError("the embedding takes an RMS norm")
            self.embed_norm = part_class("norm", spec.embed_norm.kind)(spec.embed_norm, spec.embed_norm_name)
        self.embed: Optional[torch.Tensor] = None
        self.bigram: Optional[torch.Tensor] = None
        self.position_table: Optional[torch.Tensor] = None
        self.head: Optional[Linear] = None
        self._native = None                  # the native launcher of a whole step, made at first use
        if any(getattr(b, "streams", 0) != spec.streams for b in spec.blocks):
            raise ValueError(f"the model keeps {spec.streams or 'no'} streams; every block has to keep as many")
        for e in spec.schedule:
            if not (0 <= e.block < len(self.blocks)):
                raise ValueError(f"schedule names block {e.block}, model has {len(self.blocks)}")
        self._check_cache_slots()

    # ---- what each cache slot holds ----------------------------------------------------
    def _check_cache_slots(self) -> None:
        self.kv_specs: Dict[int, KvCacheSpec] = {}
        # keyed by the cache slot (the mixer's state), by (slot, name) (a block's own) or by (MODEL, name) (the model's)
        self.state_specs: Dict[object, StateSpec] = {}
        if self.spec.bigram is not None:
            self.state_specs[(self.MODEL, "previous_token")] = StateSpec((1,), torch.int32)
        writers = set()
        for e in self.spec.schedule:
            mixer = self.blocks[e.block].mixer
            cs, ss = mixer.cache_spec(), mixer.state_spec()
            if cs is not None:
                if e.cache in self.kv_specs and self.kv_specs[e.cache] != cs:
                    raise ValueError(f"cache slot {e.cache} is used with two different layouts")
                self.kv_specs[e.cache] = cs
                if e.write_cache:
                    if e.cache in writers:
                        raise ValueError(f"cache slot {e.cache} is written by two schedule entries")
                    writers.add(e.cache)
            if ss is not None:
                if e.cache in self.state_specs and self.state_specs[e.cache] != ss:
                    raise ValueError(f"state slot {e.cache} is used with two different shapes")
                self.state_specs[e.cache] = ss
            for name, es in getattr(self.blocks[e.block], "extra_states", dict)().items():
                if self.state_specs.setdefault((e.cache, name), es) != es:
                    raise ValueError(f"state '{name}' of slot {e.cache} is used with two different shapes")
        for c in self.kv_specs:
            if c not in writers:
                raise ValueError(f"cache slot {c} is read but never written")

    # ---- weights ---------------------------------------------------------------------------
    def declare(self) -> List[TensorDecl]:
        s = self.spec
        out = [TensorDecl(s.embed_name, (s.vocab_size, s.hidden), role="embedding")]
        if s.bigram is not None:
            out.append(TensorDecl(s.bigram.name, (s.bigram.buckets + 1, s.hidden), role="embedding"))
        if s.position_table:
            out.append(TensorDecl(s.position_table, (s.max_positions, s.hidden), role="embedding"))
        if self.embed_norm is not None:
            out += self.embed_norm.declare()
        for b in self.blocks:
            out += b.declare()
        out += self.final_norm.declare()
        if not s.tie_embeddings:
            out.append(TensorDecl(s.head_name, (s.vocab_size, s.hidden)))
        seen = set()
        for d in out:
            if d.name in seen:
                raise ValueError(f"tensor '{d.name}' is declared twice")
            seen.add(d.name)
        return out

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        self.embed = tensors[s.embed_name].contiguous()
        if s.bigram is not None:
            self.bigram = tensors[s.bigram.name].to(self.embed.dtype).contiguous()
        if s.position_table:
            self.position_table = tensors[s.position_table].to(self.embed.dtype).contiguous()
        for b in self.blocks:
            b.bind(tensors)
        if self.embed_norm is not None:
            self.embed_norm.bind(tensors)
            self.embed_norm.weight = self.embed_norm.weight.float().contiguous()
        self.final_norm.bind(tensors)
        if s.logit_scale != 1.0:
            # the logits' constant multiplies what the output product reads (its norm's weight, in 32-bit)
            self.final_norm.weight = (self.final_norm.weight.float() * s.logit_scale).contiguous()
        # a tied head aliases the embedding (crates/model/src/weights.rs:2835-2849)
        self.head = Linear(self.embed if s.tie_embeddings else tensors[s.head_name], None, "lm_head")

    def weight_bytes(self) -> int:
        seen, total = set(), 0

        def add(t):
            nonlocal total
            if t is not None and t.data_ptr() not in seen:
                seen.add(t.data_ptr())
                total += t.numel() * t.element_size()
        add(self.embed)
        add(self.bigram)
        add(self.position_table)
        add(self.head.weight)
        for b in self.blocks:
            for part in b.parts():
                for v in vars(part).values():
                    if isinstance(v, Linear):
                        add(v.weight)
                        add(v.bias)
                    elif isinstance(v, torch.Tensor):
                        add(v)
        add(self.final_norm.weight)
        return total

    def _forward_streams(self, ctx, x0: torch.Tensor, logit_rows: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        """The schedule on a residual of ``spec.streams`` vectors per token (float32 [T, S, d]), all equal to the
        embedding at the start; a block returns the update of its last sublayer, which the next block applies in
        its first pass over the streams; at the end the streams are added up (on the wanted rows only)."""
        from ..kernels import layer_ops as L
        s = self.spec
        T = x0.shape[0]
        x = torch.empty((T, s.streams, s.hidden), dtype=torch.float32, device=x0.device)
        L.streams_fill(x0, x)
        pending = None
        for i, entry in enumerate(s.schedule):
            ctx.upcoming = None
            ctx.schedule_index = i
            pending = self.blocks[entry.block].forward(ctx, x, pending, entry)
        if logit_rows is None or logit_rows.numel() == 0:
            return None
        R = logit_rows.numel()
        y, mix, w_out = pending if pending is not None else (None, None, None)
        if getattr(self.final_norm.spec, "kind", "") == "layernorm":
            # the last update, the sum of the streams and the final norm of the wanted rows in one pass
            h = torch.empty((R, s.hidden), dtype=ctx.act_dtype, device=x0.device)
            L.hyper_step(x, y, mix, w_out, None, self.final_norm.weight, self.final_norm.spec.eps, h, rows=logit_rows)
        else:
            total = torch.empty((R, s.hidden), dtype=torch.float32, device=x0.device)
            L.hyper_step(x, y, mix, w_out, None, None, 0.0, None, u_out=total, rows=logit_rows)
            h = self.final_norm.forward(ctx, total, None)
        return self.head.forward(h, out_dtype=torch.float32)

    @property
    def position_limit(self) -> Optional[int]:
        """The longest sequence the model can take (None: no limit of its own): the length of its position table."""
        return self.spec.max_positions if self.spec.position_table else None

    def _embed(self, ctx, token_ids: torch.Tensor, x: torch.Tensor) -> None:
        s = self.spec
        device_tokens = getattr(ctx, "device_tokens", None)
        if s.bigram is None and not s.position_table and self.embed_norm is None:
            K.embed_gather(self.embed, token_ids, x, s.embed_scale, device_tokens)
            return
        from ..kernels import layer_ops as L
        big, previous = None, None
        if s.bigram is not None:
            big = (self.bigram, s.bigram.buckets, s.bigram.mul_prev, s.bigram.mul_cur)
            previous = ctx.state(self.MODEL, "previous_token")
        norm_w, eps, h = None, 0.0, None
        if self.embed_norm is not None:
            norm_w, eps = self.embed_norm.weight, self.embed_norm.spec.eps
        if ctx.act_dtype == torch.bfloat16 and not s.streams and s.blocks[s.schedule[0].block].kind == "postnorm":
            h = torch.empty(x.shape, dtype=torch.bfloat16, device=x.device)     # the first block reads x itself
            ctx._resid_act = (-1, h)
        L.embed_compose(self.embed, token_ids, x, s.embed_scale, device_tokens, big, previous, self.position_table, ctx.positions,
                        ctx.tok_entry, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_slot, ctx.n_entries, int(ctx.max_q_len) == 1,
                        norm_w=norm_w, eps=eps, h=h)

    # ---- one pass over the tokens of a step -------------------------------------------------
    def forward(self, ctx, token_ids: torch.Tensor, logit_rows: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        """token_ids int32 [T] on the device; logit_rows int32 [R] (indices into the T tokens)
        or None.  Returns float32 logits [R, vocab], or None when no row is wanted."""
        s = self.spec
        native = self._native
        if native is None:
            from .native_decoder import NativeDecoder
            native = self._native = NativeDecoder(self)
        out = native.run(ctx, token_ids, logit_rows)      # the whole step in one native call, where it applies
        if out is not NotImplemented:
            return out
        T = token_ids.numel()
        x = torch.empty((T, s.hidden), dtype=torch.float32, device=token_ids.device)
        self._embed(ctx, token_ids, x)
        if s.streams:
            return self._forward_streams(ctx, x, logit_rows)
        delta = None
        for i, entry in enumerate(s.schedule):
            # a block may look at what runs after it (the built-in block folds the next block's first norm
            # into its own last product when that block is of its kind)
            nxt = s.schedule[i + 1] if i + 1 < len(s.schedule) else None
            ctx.upcoming = (self.blocks[nxt.block], nxt) if nxt is not None else None
            ctx.schedule_index = i
            delta = self.blocks[entry.block].forward(ctx, x, delta, entry)
        ctx.upcoming = None
        if logit_rows is None or logit_rows.numel() == 0:
            return None
        h = self.final_norm.forward(ctx, x, delta, rows=logit_rows)
        return self.head.forward(h, out_dtype=torch.float32)
