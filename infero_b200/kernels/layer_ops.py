"""Wrappers of the kernels behind the gated post-norm block, the HGRN2 and differential-attention mixers
and the mixture-of-experts feed-forward (``csrc/gated_norm.cu``, ``hgrn2.cu``, ``diff_attention.cu``,
``moe.cu``).  Small vectors (biases, norm weights, convolution taps) are float32 on both precisions."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong
from typing import Optional

import torch

from . import _check, _dt, _i32, _ptr, _stream, lib


def _f32(t: Optional[torch.Tensor], name: str) -> Optional[torch.Tensor]:
    if t is not None and (t.dtype != torch.float32 or not t.is_contiguous()):
        raise TypeError(f"{name} must be a contiguous float32 tensor")
    return t


def cast_rows(x: torch.Tensor, out: torch.Tensor) -> None:
    """out (bf16) = x (float32), elementwise."""
    assert x.dtype == torch.float32 and out.dtype == torch.bfloat16 and x.is_contiguous() and out.is_contiguous()
    assert x.numel() == out.numel()
    _check(lib().infero_cast_rows_bf16(_ptr(x), _ptr(out), c_longlong(x.numel()), _stream()))


def gated_scalar_norm_add(x: torch.Tensor, y: torch.Tensor, gate: Optional[torch.Tensor],
                          gate_bias: Optional[torch.Tensor], norm_w: torch.Tensor, eps: float,
                          h_out: Optional[torch.Tensor] = None) -> None:
    """z = y * sigmoid(gate + gate_bias) (z = y without a gate); x += z / sqrt(mean(z^2) + eps) * norm_w[0];
    ``h_out`` (bf16) receives the new x.  x, y, gate float32 (y and gate may be column slices)."""
    T, d = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and y.shape == (T, d) and y.stride(1) == 1
    _f32(norm_w, "norm_w"), _f32(gate_bias, "gate_bias")
    assert y.dtype == torch.float32 and (gate is None or (gate.dtype == torch.float32 and gate.shape == (T, d) and gate.stride(1) == 1))
    assert h_out is None or (h_out.dtype == torch.bfloat16 and h_out.is_contiguous() and h_out.shape == (T, d))
    _check(lib().infero_gated_scalar_norm_add(_ptr(x), _ptr(y), c_int(y.stride(0)), _ptr(gate),
                                              c_int(gate.stride(0) if gate is not None else 0), _ptr(gate_bias),
                                              _ptr(norm_w), c_float(eps), _ptr(h_out), c_int(T), c_int(d), _stream()))


def hgrn2_scan(proj: torch.Tensor, q_off: int, f_off: int, v_off: int, f_bias: torch.Tensor, lower: torch.Tensor,
               out_w: torch.Tensor, eps: float, state: torch.Tensor, entry_q_start: torch.Tensor,
               entry_q_len: torch.Tensor, entry_slot: torch.Tensor, out: torch.Tensor, n_entries: int,
               H: int, D: int, V: int, q_lens=None) -> None:
    """The recurrence of every request of the step over its new tokens; see csrc/hgrn2.cu.
    proj float32 [T, >= ...] (row stride free); state float32 [slots, H, D, V]; out [T, H*V].
    ``q_lens``: the host's copy of ``entry_q_len``; with it, long portions run by chunks side by side."""
    assert proj.dtype == torch.float32 and proj.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous()
    assert tuple(state.shape[1:]) == (H, D, V) and out.shape[1] == H * V and out.stride(1) == 1
    _f32(f_bias, "f_bias"), _f32(lower, "lower"), _f32(out_w, "out_w")
    max_chunks, any_short, chunk_state, chunk_decay, chunk0 = 0, 1, None, None, None
    if q_lens is not None:
        chunk, long_ = _hgrn2_sizes()
        counts = [(-(-int(n) // chunk) if int(n) >= long_ else 0) for n in q_lens]
        max_chunks = max(counts, default=0)
        if max_chunks:
            any_short = int(any(c == 0 for c in counts))
            firsts, total = [], 0
            for c in counts:
                firsts.append(total)
                total += c
            host = torch.empty(len(firsts), dtype=torch.int32, pin_memory=True)     # (pinned: the copy is asynchronous)
            host.numpy()[:] = firsts
            chunk0 = host.to(proj.device, non_blocking=True)
            chunk_state = torch.empty((total, H, D, V), dtype=torch.float32, device=proj.device)
            chunk_decay = torch.empty((total, H, D), dtype=torch.float32, device=proj.device)
    _check(lib().infero_hgrn2_scan(_ptr(proj), c_int(proj.stride(0)), c_int(q_off), c_int(f_off), c_int(v_off),
                                   _ptr(f_bias), _ptr(lower), _ptr(out_w), c_float(eps), _ptr(state),
                                   _ptr(_i32(entry_q_start, "entry_q_start")), _ptr(_i32(entry_q_len, "entry_q_len")),
                                   _ptr(_i32(entry_slot, "entry_slot")), _ptr(out), c_int(_dt(out)), c_int(out.stride(0)),
                                   c_int(n_entries), c_int(H), c_int(D), c_int(V), c_int(max_chunks), _ptr(chunk_state),
                                   _ptr(chunk_decay), _ptr(chunk0), c_int(any_short), _stream()))


_HGRN2_SIZES = []


def _hgrn2_sizes():
    if not _HGRN2_SIZES:
        _HGRN2_SIZES.extend([int(lib().infero_hgrn2_chunk()), int(lib().infero_hgrn2_long())])
    return _HGRN2_SIZES


def qkv_prepare(proj: torch.Tensor, conv_w: Optional[torch.Tensor], taps: int, conv_state: Optional[torch.Tensor],
                q_norm: Optional[torch.Tensor], k_norm: Optional[torch.Tensor], eps: float,
                inv_freq: Optional[torch.Tensor], positions, tok_entry, entry_q_start, entry_slot, block_table,
                q_out: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, page_size: int, n_q_units: int,
                n_k_units: int, G: int, D: int, V: int, write_cache: bool = True, q_pad: bool = False) -> None:
    """Convolution over time (``conv_w`` float32 [taps, channels]), per-map RMS norm, adjacent-pair rotary, q to
    ``q_out``, k and v to their pages; see csrc/diff_attention.cu.  ``q_pad``: q_out is [T, n_q_units * 2 D], every map a query as wide as a key row
    with zeros in the other map's columns."""
    T = q_out.shape[0]
    assert q_out.shape[1] == n_q_units * D * (2 if q_pad else 1)
    assert proj.dtype == torch.float32 and proj.stride(1) == 1 and q_out.stride(1) == 1
    assert k_cache.dtype == q_out.dtype == v_cache.dtype and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert k_cache.shape[-1] == (n_k_units // G) * D and v_cache.shape[-1] == V and k_cache.shape[1] == G
    _f32(conv_w, "conv_w"), _f32(conv_state, "conv_state"), _f32(q_norm, "q_norm"), _f32(k_norm, "k_norm")
    assert conv_w is None or tuple(conv_w.shape) == (taps, (n_q_units + n_k_units) * D + G * V)
    rot = 0 if inv_freq is None else 2 * inv_freq.numel()
    _check(lib().infero_qkv_prepare(
        _ptr(proj), c_int(proj.stride(0)), _ptr(conv_w), c_int(taps), _ptr(conv_state), _ptr(q_norm), _ptr(k_norm),
        c_float(eps), _ptr(_f32(inv_freq, "inv_freq")), c_int(rot), _ptr(_i32(positions, "positions")),
        _ptr(_i32(tok_entry, "tok_entry")), _ptr(_i32(entry_q_start, "entry_q_start")),
        _ptr(_i32(entry_slot, "entry_slot")), _ptr(_i32(block_table, "block_table")), c_int(block_table.shape[1]),
        _ptr(q_out), c_int(q_out.stride(0)), _ptr(k_cache), _ptr(v_cache), c_int(_dt(q_out)), c_int(page_size),
        c_int(T), c_int(n_q_units), c_int(n_k_units), c_int(G), c_int(D), c_int(V), c_int(1 if write_cache else 0),
        c_int(1 if q_pad else 0), _stream()))


def diff_combine(maps: torch.Tensor, out: torch.Tensor, H: int, V: int, lam: float, eps: float, out_scale: float) -> None:
    """maps [T, H*2*V] (per head the two maps' attention results) -> out [T, H*V]: a1 - lam a2, weightless RMS norm
    over V, times out_scale."""
    T = maps.shape[0]
    assert maps.dtype == out.dtype and maps.stride(1) == 1 and out.stride(1) == 1 and maps.shape[1] == 2 * H * V
    _check(lib().infero_diff_combine(_ptr(maps), c_int(maps.stride(0)), _ptr(out), c_int(out.stride(0)), c_int(_dt(out)),
                                     c_int(T), c_int(H), c_int(V), c_float(lam), c_float(eps), c_float(out_scale), _stream()))


def conv_state_update(proj: torch.Tensor, conv_state: torch.Tensor, taps: int, entry_q_start, entry_q_len,
                      entry_slot, n_entries: int, channels: int) -> None:
    """The last taps - 1 product rows of every request become its state (float32 [slots, taps-1, channels])."""
    assert conv_state.dtype == torch.float32 and conv_state.is_contiguous()
    assert tuple(conv_state.shape[1:]) == (taps - 1, channels)
    _check(lib().infero_conv_state_update(_ptr(proj), c_int(proj.stride(0)), _ptr(conv_state), c_int(taps),
                                          _ptr(_i32(entry_q_start, "entry_q_start")),
                                          _ptr(_i32(entry_q_len, "entry_q_len")), _ptr(_i32(entry_slot, "entry_slot")),
                                          c_int(n_entries), c_int(channels), _stream()))


def diff_attention_generic(q, out, k_cache, v_cache, block_table, tok_entry, positions, H: int, G: int, D: int,
                           V: int, page_size: int, window: Optional[int], scale: float, lam: float, eps: float,
                           out_scale: float) -> None:
    """One warp per (token, head): two causal softmaxes over the same values, a1 - lam a2, weightless RMS
    norm over V, times out_scale.  q [T, H*2*D], out [T, H*V], caches of q's dtype."""
    T = q.shape[0]
    assert q.stride(1) == 1 and out.stride(1) == 1 and q.dtype == out.dtype == k_cache.dtype == v_cache.dtype
    _check(lib().infero_diff_attention_generic(
        _ptr(q), c_int(q.stride(0)), _ptr(out), c_int(out.stride(0)), _ptr(k_cache), _ptr(v_cache), c_int(_dt(q)),
        _ptr(_i32(block_table, "block_table")), c_int(block_table.shape[1]), _ptr(_i32(tok_entry, "tok_entry")),
        _ptr(_i32(positions, "positions")), c_int(T), c_int(H), c_int(G), c_int(D), c_int(V), c_int(page_size),
        c_int(window or 0), c_float(scale), c_float(lam), c_float(eps), c_float(out_scale), _stream()))


def moe_select(logits: torch.Tensor, E: int, top: int, gate_col: int = -1):
    """From float32 logits [T, >= E] (row stride free): (top_idx int32 [T, top], top_w float32 [T, top], gate float32
    [T] or None): the ``top`` largest of the first E columns, softmax over those alone; gate = sigmoid(column
    ``gate_col``).  See csrc/moe.cu."""
    T = logits.shape[0]
    assert logits.dtype == torch.float32 and logits.stride(1) == 1 and logits.shape[1] >= E
    idx = torch.empty((T, top), dtype=torch.int32, device=logits.device)
    w = torch.empty((T, top), dtype=torch.float32, device=logits.device)
    gate = torch.empty(T, dtype=torch.float32, device=logits.device) if gate_col >= 0 else None
    _check(lib().infero_moe_select(_ptr(logits), c_int(logits.stride(0)), c_int(gate_col), _ptr(idx), _ptr(w), _ptr(gate),
                                   c_int(T), c_int(E), c_int(top), _stream()))
    return idx, w, gate


GLU_KINDS = {"swiglu": 0, "glu_clamped": 1}


def _act_args(act):
    """(kind, limit, alpha) of a gated activation as the kernels take it; None: silu(g) * u."""
    if act is None:
        return c_int(0), c_float(0.0), c_float(1.0)
    kind, limit, alpha = act
    return c_int(GLU_KINDS[kind]), c_float(limit), c_float(alpha)


def moe_experts_streamed(h, gate_up, down, top_idx, top_w, shared, shared_gate, y, act=None) -> None:
    """y[t] = sum_c top_w[t, c] * expert_{top_idx[t, c]}(h[t]) (+ shared_gate[t] * shared[t]); every (token,
    choice) streams its expert's rows.  gate_up [E, 2 ff, d] (rows alternate gate_j, up_j), down [E, d, ff]."""
    T, d = h.shape
    E, ff2, _ = gate_up.shape
    ff, top = ff2 // 2, top_idx.shape[1]
    assert gate_up.dtype == h.dtype == down.dtype and gate_up.is_contiguous() and down.is_contiguous()
    assert tuple(down.shape) == (E, d, ff) and y.dtype == torch.float32 and y.is_contiguous() and y.shape == (T, d)
    scratch = torch.empty((T * top, ff), dtype=h.dtype, device=h.device)
    _check(lib().infero_moe_experts_streamed(_ptr(h), c_int(h.stride(0)), _ptr(gate_up), _ptr(down), c_int(_dt(h)),
                                             _ptr(_i32(top_idx, "top_idx")), _ptr(_f32(top_w, "top_w")),
                                             _ptr(_f32(shared, "shared")), _ptr(_f32(shared_gate, "shared_gate")),
                                             _ptr(scratch), _ptr(y), c_int(T), c_int(d), c_int(ff), c_int(top),
                                             *_act_args(act), _stream()))


def moe_experts_grouped(h, gate_up, down, top_idx, top_w, shared, shared_gate, y, act=None) -> None:
    """The same result as ``moe_experts_streamed`` by grouped tensor-core products (bf16): the (token, choice)
    pairs are sorted by expert into 64-row tiles; see csrc/moe_grouped.cu."""
    T, d = h.shape
    E, ff2, _ = gate_up.shape
    ff, top = ff2 // 2, top_idx.shape[1]
    assert h.dtype == torch.bfloat16 and gate_up.dtype == torch.bfloat16 and down.dtype == torch.bfloat16
    assert gate_up.is_contiguous() and down.is_contiguous() and tuple(down.shape) == (E, d, ff)
    assert y.dtype == torch.float32 and y.is_contiguous() and y.shape == (T, d) and h.stride(1) == 1
    tiles = int(lib().infero_moe_grouped_tiles(c_int(T * top), c_int(E)))
    R = tiles * int(lib().infero_moe_grouped_tile_rows(c_int(T * top), c_int(E)))
    dev = h.device
    ints = torch.empty(2 * R + tiles + 1, dtype=torch.int32, device=dev)
    sorted_pair, a_rows, tile_expert = ints[:R], ints[R:2 * R], ints[2 * R:]
    scratch = torch.empty((R, ff), dtype=torch.bfloat16, device=dev)
    part = torch.empty((T * top, d), dtype=torch.float32, device=dev)
    _check(lib().infero_moe_experts_grouped(_ptr(h), c_int(h.stride(0)), _ptr(gate_up), _ptr(down),
                                            _ptr(_i32(top_idx, "top_idx")), _ptr(_f32(top_w, "top_w")),
                                            _ptr(_f32(shared, "shared")), _ptr(_f32(shared_gate, "shared_gate")),
                                            _ptr(sorted_pair), _ptr(a_rows), _ptr(tile_expert), _ptr(scratch), _ptr(part),
                                            _ptr(y), c_int(T), c_int(d), c_int(ff), c_int(E), c_int(top), *_act_args(act),
                                            _stream()))


def moe_experts_tc(h, gate_up, down, top_idx, top_w, shared, shared_gate, y, act=None) -> None:
    """The same result by grouped products on the tcgen05 kernel: the tokens' rows are copied into expert order in
    tiles of 128 rows, two grouped products (the first with the SwiGLU epilogue) run over them, and the rows of a
    token's choices are added up in ascending order; see csrc/moe_grouped.cu and ``infero_gemm_tc_grouped``."""
    from .tc_gemm import sm_count
    T, d = h.shape
    E, ff2, _ = gate_up.shape
    ff, top = ff2 // 2, top_idx.shape[1]
    assert h.dtype == torch.bfloat16 and gate_up.dtype == torch.bfloat16 and down.dtype == torch.bfloat16
    assert gate_up.is_contiguous() and down.is_contiguous() and tuple(down.shape) == (E, d, ff)
    assert y.dtype == torch.float32 and y.is_contiguous() and y.shape == (T, d) and h.stride(1) == 1
    tiles = int(lib().infero_moe_tc_tiles(c_int(T * top), c_int(E)))
    R, dev = tiles * 128, h.device
    ints = torch.empty(2 * R + tiles + 1 + T * top, dtype=torch.int32, device=dev)
    sorted_pair, a_rows, tile_expert, pair_row = ints[:R], ints[R:2 * R], ints[2 * R:2 * R + tiles + 1], ints[2 * R + tiles + 1:]
    xs = torch.empty((R, d), dtype=torch.bfloat16, device=dev)
    _check(lib().infero_moe_tc_prepare(_ptr(h), c_int(h.stride(0)), _ptr(_i32(top_idx, "top_idx")), _ptr(sorted_pair),
                                       _ptr(a_rows), _ptr(tile_expert), _ptr(pair_row), _ptr(xs), c_int(T), c_int(d),
                                       c_int(E), c_int(top), _stream()))
    scratch = torch.empty((R, ff), dtype=torch.bfloat16, device=dev)
    sms = sm_count(dev)
    _check(lib().infero_gemm_tc_grouped(_ptr(xs), _ptr(gate_up), _ptr(scratch), c_int(1), c_int(R), c_int(2 * ff), c_int(d),
                                        c_int(d), c_int(ff), _ptr(tile_expert), c_int(E), c_int(sms), *_act_args(act),
                                        _stream()))
    rows = torch.empty((R, d), dtype=torch.float32, device=dev)
    _check(lib().infero_gemm_tc_grouped(_ptr(scratch), _ptr(down), _ptr(rows), c_int(0), c_int(R), c_int(d), c_int(ff),
                                        c_int(ff), c_int(d), _ptr(tile_expert), c_int(E), c_int(sms), *_act_args(None),
                                        _stream()))
    _check(lib().infero_moe_tc_combine(_ptr(rows), _ptr(pair_row), _ptr(_f32(top_w, "top_w")), _ptr(_f32(shared, "shared")),
                                       _ptr(_f32(shared_gate, "shared_gate")), _ptr(y), c_int(T), c_int(d), c_int(top),
                                       _stream()))


def moe_select_grouped(logits: torch.Tensor, correction: Optional[torch.Tensor], E: int, top: int, groups: int = 1,
                       keep: int = 1):
    """From float32 logits [T, >= E]: s = softmax over the E experts; the ``top`` largest of s + correction among the
    ``keep`` best of ``groups`` groups of neighbouring experts; (top_idx int32 [T, top], top_w float32 [T, top]) with
    top_w = s of the chosen over their sum.  See csrc/moe.cu."""
    T = logits.shape[0]
    assert logits.dtype == torch.float32 and logits.stride(1) == 1 and logits.shape[1] >= E
    assert correction is None or correction.numel() == E
    idx = torch.empty((T, top), dtype=torch.int32, device=logits.device)
    w = torch.empty((T, top), dtype=torch.float32, device=logits.device)
    _check(lib().infero_moe_select_grouped(_ptr(logits), c_int(logits.stride(0)), _ptr(_f32(correction, "correction")),
                                           _ptr(idx), _ptr(w), c_int(T), c_int(E), c_int(top), c_int(groups), c_int(keep),
                                           _stream()))
    return idx, w


def _product_in(v):
    """(pointer source, dtype tag, splits, split stride, shape) of a product given as a tensor or as partial sums."""
    from . import Partials
    if isinstance(v, Partials):
        assert v.bias is None
        return v.data, 0, v.splits, v.split_stride, tuple(v.shape)
    assert v.is_contiguous()
    return v, _dt(v), 1, 0, tuple(v.shape)


def glu_act(gate_up, out: torch.Tensor, act=None, bias: Optional[torch.Tensor] = None) -> None:
    """out[t, j] = glu(g[t, 2j], g[t, 2j + 1]) for g = gate_up (a tensor or ``Partials``; gate and up alternate along a
    row); ``act`` = (kind, limit, alpha), None: silu(g) * u; ``bias`` float32 [2 ff] is added to g first (``Partials`` bring
    their own)."""
    T, ff = out.shape
    if getattr(gate_up, "bias", None) is not None:
        from . import Partials
        assert bias is None
        gate_up, bias = Partials(gate_up.data), gate_up.bias
    assert bias is None or bias.numel() == 2 * ff
    data, dt, splits, stride, shape = _product_in(gate_up)
    assert shape == (T, 2 * ff) and out.is_contiguous()
    _check(lib().infero_glu_act(_ptr(data), c_int(dt), c_int(splits), c_longlong(stride), _ptr(out), c_int(_dt(out)), c_int(T),
                                c_int(ff), *_act_args(act), _ptr(_f32(bias, "bias")), _stream()))


def relu2(v, out: torch.Tensor) -> None:
    """out = max(v, 0)^2, v a tensor or ``Partials`` of out's shape."""
    T, ff = out.shape
    data, dt, splits, stride, shape = _product_in(v)
    assert shape == (T, ff) and out.is_contiguous()
    _check(lib().infero_relu2(_ptr(data), c_int(dt), c_int(splits), c_longlong(stride), _ptr(out), c_int(_dt(out)), c_int(T),
                              c_int(ff), _stream()))


def add_layernorm(x: torch.Tensor, delta: Optional[torch.Tensor], weight: torch.Tensor, eps: float, out: torch.Tensor,
                  rows: Optional[torch.Tensor] = None) -> None:
    """x += delta (float32, if given); out = layer norm of x (weight, no bias).  With ``rows`` only those rows are
    normalised and x is left as it is."""
    d = x.shape[1]
    assert x.dtype == torch.float32 and x.is_contiguous() and out.is_contiguous() and out.shape[1] == d
    assert delta is None or (delta.dtype == torch.float32 and delta.is_contiguous() and delta.shape == x.shape)
    n = out.shape[0]
    assert n == (x.shape[0] if rows is None else rows.numel()) and weight.numel() == d
    _check(lib().infero_add_layernorm(_ptr(x), _ptr(delta), _ptr(_f32(weight, "weight")), c_float(eps), _ptr(out),
                                      c_int(_dt(out)), _ptr(None if rows is None else _i32(rows, "rows")), c_int(n), c_int(d),
                                      _stream()))


def hyper_step(xs: torch.Tensor, y, mix: Optional[torch.Tensor], w_out: Optional[torch.Tensor],
               w_in: Optional[torch.Tensor], norm_w: Optional[torch.Tensor], eps: float, h_out: Optional[torch.Tensor],
               u_out: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None) -> None:
    """One pass over the streams xs (float32 [T, S, d]) of every token: with ``y`` (float32 [T, d], or a product left as
    ``Partials``) the update xs[r] <- sum_s mix[s, r] xs[s] + w_out[r] y; with ``w_in`` and ``norm_w`` the next
    sublayer's input h_out = layer norm(sum_s w_in[s] xs[s]); with ``u_out`` (float32) and no norm the weighted sum itself
    (w_in None: the plain sum).  ``rows``: work on these tokens only."""
    from . import Partials
    T, S, d = xs.shape
    assert xs.dtype == torch.float32 and xs.is_contiguous()
    splits, split_stride, y_stride = 1, 0, 0
    if isinstance(y, Partials):
        assert y.bias is None and tuple(y.shape) == (T, d)
        y, splits, split_stride, y_stride = y.data, y.splits, y.split_stride, d
    elif y is not None:
        assert y.dtype == torch.float32 and y.shape == (T, d) and y.stride(1) == 1
        y_stride = y.stride(0)
    n = T if rows is None else rows.numel()
    for o in (h_out, u_out):
        assert o is None or (o.is_contiguous() and tuple(o.shape) == (n, d))
    assert u_out is None or u_out.dtype == torch.float32
    _check(lib().infero_hyper_step(_ptr(xs), _ptr(y), c_int(y_stride), c_int(splits), c_longlong(split_stride),
                                   _ptr(_f32(mix, "mix")), _ptr(_f32(w_out, "w_out")), _ptr(_f32(w_in, "w_in")),
                                   _ptr(_f32(norm_w, "norm_w")), c_float(eps), _ptr(h_out),
                                   c_int(_dt(h_out) if h_out is not None else 0), _ptr(u_out),
                                   _ptr(None if rows is None else _i32(rows, "rows")), c_int(n), c_int(S), c_int(d), _stream()))


def streams_fill(x: torch.Tensor, xs: torch.Tensor) -> None:
    """xs[t, s] = x[t] for every stream s."""
    T, S, d = xs.shape
    assert x.dtype == xs.dtype == torch.float32 and x.is_contiguous() and xs.is_contiguous() and tuple(x.shape) == (T, d)
    _check(lib().infero_streams_fill(_ptr(x), _ptr(xs), c_int(T), c_int(S), c_int(d), _stream()))


# ---- normed attention, gated linear recurrence (csrc/qk_prepare.cu, rglru.cu) ------------------------------------
def qk_prepare(proj: torch.Tensor, q_off: int, k_off: int, v_off: int, norm_mode: int, q_norm_w, k_norm_w, eps: float,
               freq64: Optional[torch.Tensor], amp: float, positions, tok_entry, block_table, page_size: int,
               q_out: torch.Tensor, k_cache, v_cache, H: int, G: int, D: int, V: int, write_cache: bool = True,
               temperature=None, v_scale: float = 1.0) -> None:
    """From the 32-bit product row of every token (``proj`` [T, >= ...], columns ``q_off`` / ``k_off`` / ``v_off``; a
    negative ``v_off``: the values are the keys as projected) to normed, rotated queries in ``q_out`` [T, H*D] and keys and
    values in the token's page.  ``norm_mode`` 0 none, 1 weighted RMS over the whole projection before the rotation,
    2 unit RMS per head after it, 3 weighted RMS per head before it (weights of D numbers shared by the heads).
    ``freq64`` float64 [rot/2] (None: no rotation), ``amp`` multiplies cos and sin.  ``temperature`` = (coef, every): a
    query at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1) at the end.  ``v_scale`` multiplies values
    of a projection of their own."""
    T = proj.shape[0]
    assert proj.dtype == torch.float32 and proj.stride(1) == 1 and q_out.stride(1) == 1 and q_out.shape == (T, H * D)
    rot = 0
    if freq64 is not None:
        assert freq64.dtype == torch.float64 and freq64.is_contiguous()
        rot = 2 * freq64.numel()
    if write_cache:
        assert k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.dtype == q_out.dtype == v_cache.dtype
        assert k_cache.shape[1:] == (G, page_size, D) and v_cache.shape[1:] == (G, page_size, V)
    if norm_mode == 1:
        assert q_norm_w.numel() == H * D and (not write_cache or k_norm_w.numel() == G * D)
        assert k_norm_w is None or k_norm_w.dtype == q_norm_w.dtype
    if norm_mode == 3:
        assert q_norm_w.numel() == D and (not write_cache or k_norm_w.numel() == D)
        assert k_norm_w is None or k_norm_w.dtype == q_norm_w.dtype
    _check(lib().infero_qk_prepare(
        _ptr(proj), c_int(proj.stride(0)), c_int(q_off), c_int(k_off), c_int(v_off), c_int(norm_mode), _ptr(q_norm_w),
        _ptr(k_norm_w), c_int(_dt(q_norm_w) if q_norm_w is not None else 0), c_float(eps), _ptr(freq64), c_int(rot),
        c_float(amp), _ptr(_i32(positions, "positions")), _ptr(_i32(tok_entry, "tok_entry")),
        _ptr(_i32(block_table, "block_table")), c_int(block_table.shape[1]), c_int(page_size), _ptr(q_out),
        c_int(q_out.stride(0)), _ptr(k_cache if write_cache else None), _ptr(v_cache if write_cache else None),
        c_int(_dt(q_out)), c_int(1 if write_cache else 0), c_int(T), c_int(H), c_int(G), c_int(D), c_int(V),
        c_float(temperature[0] if temperature else 0.0), c_float(temperature[1] if temperature else 0.0), c_float(v_scale), _stream()))


def head_gate(a: torch.Tensor, gate: Optional[torch.Tensor], out: torch.Tensor, H: int, V: int, scale: float = 1.0) -> None:
    """out[t, h*V + v] = a[t, h*V + v] * sigmoid(gate[t, h]) * scale (no gate: only the factor); gate float32, a column
    slice allowed; ``out`` may be ``a`` or a column slice of a wider array."""
    T = a.shape[0]
    assert a.shape == (T, H * V) and out.shape == (T, H * V) and a.stride(1) == 1 and out.stride(1) == 1 and a.dtype == out.dtype
    assert gate is None or (gate.dtype == torch.float32 and gate.shape == (T, H) and gate.stride(1) == 1)
    _check(lib().infero_head_gate(_ptr(a), c_int(a.stride(0)), _ptr(gate), c_int(gate.stride(0) if gate is not None else 0),
                                  _ptr(out), c_int(out.stride(0)), c_int(_dt(a)), c_int(T), c_int(H), c_int(V), c_float(scale),
                                  _stream()))


def rglru(proj: torch.Tensor, y_off: int, x_off: int, conv_w: torch.Tensor, conv_b: Optional[torch.Tensor], w_gates: torch.Tensor,
          ra_b: torch.Tensor, ri_b: torch.Tensor, lam: torch.Tensor, slope: float, state: torch.Tensor, tok_entry,
          entry_q_start, entry_q_len, entry_slot, n_entries: int, out: torch.Tensor, scale: float = 1.0,
          max_q_len: int = 1, tensor_cores: bool = False, conv_wt: Optional[torch.Tensor] = None) -> None:
    """The gated linear recurrence of every request of the step over its new tokens; see csrc/rglru.cu.  ``proj`` float32
    [T, >= ...] holds the gate branch at ``y_off`` and the recurrent branch at ``x_off`` (C columns each, biases added);
    ``conv_w`` float32 [C, taps]; ``w_gates`` [blocks, 2 C/blocks, C/blocks] (float32 or bf16): per block the rows of Ra,
    then those of Ri; ``state`` float32 [slots, taps, C] (rows 0..taps-2 the convolution's last inputs, row taps-1 the
    recurrent state); ``out`` [T, C] (a column slice allowed) receives S * gelu_tanh(y) * scale.  ``max_q_len``: the
    longest portion of the step.  ``tensor_cores``: the gate products of a long bf16 step run as one grouped
    tensor-core product over all blocks, from u rounded to bf16 (32-bit sums); otherwise they are 32-bit throughout.
    ``conv_wt``: ``conv_w`` laid out tap-major, float32 [taps, C], as the kernels read it (made here when absent)."""
    T = proj.shape[0]
    C, taps = conv_w.shape
    blocks, two_bs, bs = w_gates.shape
    assert proj.dtype == torch.float32 and proj.stride(1) == 1 and out.shape == (T, C) and out.stride(1) == 1
    assert state.dtype == torch.float32 and state.is_contiguous() and tuple(state.shape[1:]) == (taps, C)
    assert blocks * bs == C and two_bs == 2 * bs and w_gates.is_contiguous()
    _f32(conv_w, "conv_w"), _f32(conv_b, "conv_b"), _f32(ra_b, "ra_b"), _f32(ri_b, "ri_b"), _f32(lam, "lam")
    if conv_wt is None:
        conv_wt = conv_w.t().contiguous()
    assert conv_wt.dtype == torch.float32 and conv_wt.is_contiguous() and tuple(conv_wt.shape) == (taps, C)
    L = lib()
    if int(max_q_len) == 1 and w_gates.dtype == torch.bfloat16 and bs % 8 == 0 and bs <= 256:
        # a step of single tokens: one launch for convolution, gate products and the state's update
        rc = L.infero_rglru_step(_ptr(proj), c_int(proj.stride(0)), c_int(y_off), c_int(x_off), _ptr(conv_wt), _ptr(conv_b),
                                 c_int(taps), _ptr(w_gates), _ptr(ra_b), _ptr(ri_b), _ptr(lam), c_float(slope), _ptr(state),
                                 _ptr(_i32(entry_q_start, "entry_q_start")), _ptr(_i32(entry_q_len, "entry_q_len")),
                                 _ptr(_i32(entry_slot, "entry_slot")), _ptr(out), c_int(out.stride(0)), c_int(_dt(out)),
                                 c_int(n_entries), c_int(C), c_int(blocks), c_float(scale), _stream())
        if rc != 2:
            _check(rc)
            return
    u = torch.empty((T, C), dtype=torch.float32, device=proj.device)
    u16 = None
    rows = -(-T // 128) * 128
    if tensor_cores and T > 256 and w_gates.dtype == torch.bfloat16:
        from . import latent_attention as LA
        u16 = torch.empty((blocks, rows, bs), dtype=torch.bfloat16, device=proj.device)
        if not LA.grouped_ok(u16, w_gates):
            u16 = None
    _check(L.infero_rglru_conv(_ptr(proj), c_int(proj.stride(0)), c_int(x_off), _ptr(conv_wt), _ptr(conv_b), c_int(taps),
                               _ptr(state), _ptr(_i32(tok_entry, "tok_entry")), _ptr(_i32(entry_q_start, "entry_q_start")),
                               _ptr(_i32(entry_slot, "entry_slot")), _ptr(u), _ptr(u16), c_int(blocks), c_longlong(rows), c_int(T),
                               c_int(C), _stream()))
    if u16 is not None:
        # one grouped product over all blocks: [blocks, rows, bs] x [blocks, 2 bs, bs]^T -> [blocks, rows, 2 bs]
        gates = torch.empty((blocks, rows, 2 * bs), dtype=torch.float32, device=proj.device)
        LA.per_head_product(u16, w_gates, gates, T)
        g_tok, g_blk = 2 * bs, rows * 2 * bs
    else:
        gates = torch.empty((T, 2 * C), dtype=torch.float32, device=proj.device)
        _check(L.infero_rglru_gates(_ptr(u), _ptr(w_gates), c_int(_dt(w_gates)), _ptr(gates), c_int(T), c_int(C), c_int(blocks),
                                    _stream()))
        g_tok, g_blk = 2 * C, 2 * bs
    _check(L.infero_rglru_scan(_ptr(proj), c_int(proj.stride(0)), c_int(y_off), c_int(x_off), _ptr(u), _ptr(gates),
                               c_longlong(g_tok), c_longlong(g_blk), _ptr(ra_b), _ptr(ri_b), _ptr(lam), c_float(slope),
                               c_int(taps), _ptr(state), _ptr(_i32(entry_q_start, "entry_q_start")),
                               _ptr(_i32(entry_q_len, "entry_q_len")), _ptr(_i32(entry_slot, "entry_slot")), _ptr(out),
                               c_int(out.stride(0)), c_int(_dt(out)),
                               c_int(n_entries), c_int(C), c_int(blocks), c_int(max(1, int(max_q_len))), c_float(scale), _stream()))


# ---- state-space recurrence (csrc/ssd.cu), gated group norm ---------------------------------------------------------
def ssd_state_floats(heads: int, N: int, P: int, groups: int, taps: int) -> int:
    """Floats of one request's state: the convolution's last taps - 1 inputs, then S [heads, N, P]."""
    return (taps - 1) * (heads * P + 2 * groups * N) + heads * N * P


def ssd(proj: torch.Tensor, z_off: int, x_off: int, dt_off: int, conv_w: torch.Tensor, conv_b: Optional[torch.Tensor],
        dt_bias: torch.Tensor, a_log: torch.Tensor, skip: torch.Tensor, norm_w: torch.Tensor, eps: float, norm_groups: int,
        state: torch.Tensor, tok_entry, entry_q_start, entry_q_len, entry_slot, n_entries: int, out: torch.Tensor,
        heads: int, groups: int, N: int, P: int, scale: float = 1.0, max_q_len: int = 1) -> None:
    """The state-space recurrence of every request of the step over its new tokens, and the gated, grouped norm of its
    result; see csrc/ssd.cu.  ``proj`` float32 [T, >= ...] holds [z | x B C | dt] at ``z_off`` / ``x_off`` / ``dt_off``;
    ``conv_w`` float32 [CH, taps] over the CH = heads P + 2 groups N channels of [x | B | C]; ``state`` float32
    [slots, floats] (``ssd_state_floats``); ``out`` [T, heads * P] (a column slice allowed) receives
    rms_parts(y * silu(z)) * norm_w * scale.  ``max_q_len``: the longest portion of the step."""
    from .tc_gemm import sm_count
    T = proj.shape[0]
    CH, taps = conv_w.shape
    inner = heads * P
    assert CH == inner + 2 * groups * N and proj.dtype == torch.float32 and proj.stride(1) == 1
    assert out.shape == (T, inner) and out.stride(1) == 1
    assert state.dtype == torch.float32 and state.is_contiguous() and state.shape[1] == ssd_state_floats(heads, N, P, groups, taps)
    _f32(conv_w, "conv_w"), _f32(conv_b, "conv_b"), _f32(dt_bias, "dt_bias"), _f32(a_log, "a_log"), _f32(skip, "skip"), _f32(norm_w, "norm_w")
    dev = proj.device
    L = lib()
    u = torch.empty((T, CH), dtype=torch.float32, device=dev)
    qs, ql, sl = _ptr(_i32(entry_q_start, "entry_q_start")), _ptr(_i32(entry_q_len, "entry_q_len")), _ptr(_i32(entry_slot, "entry_slot"))
    _check(L.infero_ssd_conv(_ptr(proj), c_int(proj.stride(0)), c_int(x_off), _ptr(conv_w), _ptr(conv_b), c_int(taps), _ptr(state),
                             c_longlong(state.stride(0)), _ptr(_i32(tok_entry, "tok_entry")), qs, ql, sl, _ptr(u), c_int(T),
                             c_int(n_entries), c_int(CH), _stream()))
    y = torch.empty((T, inner), dtype=torch.float32, device=dev)
    L.infero_ssd_scan_scratch.restype = c_longlong
    need = int(L.infero_ssd_scan_scratch(c_int(n_entries), c_int(int(max_q_len)), c_int(heads), c_int(N), c_int(P)))
    scratch = torch.empty(need, dtype=torch.float32, device=dev) if need else None
    _check(L.infero_ssd_scan(_ptr(u), _ptr(proj), c_int(proj.stride(0)), c_int(dt_off), _ptr(dt_bias), _ptr(a_log), _ptr(skip),
                             _ptr(state), c_longlong(state.stride(0)), c_int(taps), qs, ql, sl, _ptr(y), c_int(n_entries),
                             c_int(max(1, int(max_q_len))), c_int(heads), c_int(groups), c_int(N), c_int(P), _ptr(scratch),
                             c_int(sm_count(dev)), _stream()))
    gated_group_norm(y, proj[:, z_off:z_off + inner], norm_w, eps, norm_groups, out, scale)


def gated_group_norm(y: torch.Tensor, gate: Optional[torch.Tensor], weight: torch.Tensor, eps: float, parts: int,
                     out: torch.Tensor, scale: float = 1.0) -> None:
    """out = v / sqrt(mean over each of ``parts`` equal parts of v^2 + eps) * weight * scale with v = y * silu(gate)
    (v = y without a gate).  y, gate float32 [T, n] (column slices allowed); out [T, n] of any element type."""
    T, n = y.shape
    assert y.dtype == torch.float32 and y.stride(1) == 1 and out.shape == (T, n) and out.stride(1) == 1
    assert gate is None or (gate.dtype == torch.float32 and gate.shape == (T, n) and gate.stride(1) == 1)
    assert weight.numel() == n
    _check(lib().infero_gated_group_norm(_ptr(y), c_int(y.stride(0)), _ptr(gate), c_int(gate.stride(0) if gate is not None else 0),
                                         _ptr(_f32(weight, "weight")), c_float(eps), c_float(scale), _ptr(out),
                                         c_int(out.stride(0)), c_int(_dt(out)), c_int(T), c_int(n), c_int(parts), _stream()))


# ---- norms around a sublayer, input convolution (csrc/sandwich_norm.cu) --------------------------------------------
def _branch(v, shape):
    """(data, splits, split stride, bias) of a 32-bit sublayer result given as a tensor or as partial sums."""
    from . import Partials
    if v is None:
        return None, 1, 0, None
    if isinstance(v, Partials):
        assert tuple(v.shape) == tuple(shape)
        return v.data, v.splits, v.split_stride, _f32(v.bias, "bias")
    assert v.dtype == torch.float32 and v.is_contiguous() and tuple(v.shape) == tuple(shape)
    return v, 1, 0, None


def sandwich_norm(x: torch.Tensor, delta, weight: Optional[torch.Tensor], eps: float, out: Optional[torch.Tensor],
                  rows: Optional[torch.Tensor] = None, conv=None) -> None:
    """x += rms(z) * w for a pending ``NormedDelta`` (None: x is left as it is; a plain 32-bit tensor or ``Partials`` is
    added as it is), then out = rms(x) * weight (no weight: out = x; no out: nothing more).  With ``rows`` only those rows are worked on and x is left as it is.
    ``conv`` = (weights [taps, d], state [slots, (taps - 1) d], tok_entry, entry_slot): in a step of single tokens, out
    becomes out + the convolution of it over the requests' earlier rows, and the state moves on."""
    from . import BranchSum, NormedDelta
    d = x.shape[1]
    assert x.dtype == torch.float32 and x.is_contiguous() and (out is None or (out.is_contiguous() and out.shape[1] == d))
    n = x.shape[0] if rows is None else rows.numel()
    assert out is None or out.shape[0] == n
    assert weight is None or weight.numel() == d
    w_post, post_eps, value = None, 0.0, delta
    if isinstance(delta, NormedDelta):
        w_post, post_eps, value = _f32(delta.weight, "weight"), delta.eps, delta.value
        assert w_post.numel() == d
    second, w0, w1, scale, branch_eps = None, None, None, 1.0, 0.0
    if isinstance(value, BranchSum):
        (value, second), (w0, w1), scale, branch_eps = value.values, value.weights, value.scale, value.eps
        assert w0.numel() == d and w1.numel() == d
    y0, s0, st0, b0 = _branch(value, x.shape)
    y1, s1, st1, b1 = _branch(second, x.shape)
    cw, taps, state, stride, tok_entry, entry_slot = None, 0, None, 0, None, None
    if conv is not None:
        cw, state, tok_entry, entry_slot = conv
        taps = cw.shape[0]
        assert tuple(cw.shape) == (taps, d) and state.dtype == torch.float32 and state.is_contiguous()
        assert state.shape[1] == (taps - 1) * d or taps == 1
        stride = state.stride(0)
    _check(lib().infero_sandwich_norm(
        _ptr(x), _ptr(y0), c_int(s0), c_longlong(st0), _ptr(b0), _ptr(_f32(w0, "w0")), _ptr(y1), c_int(s1), c_longlong(st1),
        _ptr(b1), _ptr(_f32(w1, "w1")), c_float(scale), c_float(branch_eps), _ptr(w_post), c_float(post_eps),
        _ptr(_f32(weight, "weight")), c_float(eps), _ptr(out), c_int(_dt(out) if out is not None else 0),
        _ptr(None if rows is None else _i32(rows, "rows")), c_int(n), c_int(d), _ptr(_f32(cw, "conv")), c_int(taps), _ptr(state),
        c_longlong(stride), _ptr(tok_entry), _ptr(entry_slot), _stream()))


def input_conv(h: torch.Tensor, w: torch.Tensor, state: torch.Tensor, tok_entry, entry_q_start, entry_q_len, entry_slot,
               n_entries: int, out: torch.Tensor) -> None:
    """out = h + the causal convolution of h over time, per channel; then the requests' states move on.  h float32 [T, d],
    w float32 [taps, d], state float32 [slots, (taps - 1) d]."""
    T, d = h.shape
    taps = w.shape[0]
    assert h.dtype == torch.float32 and h.is_contiguous() and out.is_contiguous() and out.shape == h.shape and w.shape[1] == d
    assert state.dtype == torch.float32 and state.is_contiguous() and (taps == 1 or state.shape[1] == (taps - 1) * d)
    _check(lib().infero_input_conv(_ptr(h), _ptr(_f32(w, "w")), c_int(taps), _ptr(state), c_longlong(state.stride(0)),
                                   _ptr(_i32(tok_entry, "tok_entry")), _ptr(_i32(entry_q_start, "entry_q_start")),
                                   _ptr(_i32(entry_q_len, "entry_q_len")), _ptr(_i32(entry_slot, "entry_slot")), _ptr(out),
                                   c_int(_dt(out)), c_int(T), c_int(n_entries), c_int(d), _stream()))


# ---- embedding of a token, of its pair with the one before, and of its position (csrc/embed_compose.cu) -----------
def embed_compose(table: torch.Tensor, ids: torch.Tensor, out_x: torch.Tensor, scale: float, device_tokens, bigram, previous,
                  pos_table, positions, tok_entry, entry_q_start, entry_q_len, entry_slot, n_entries: int, single: bool,
                  norm_w: Optional[torch.Tensor] = None, eps: float = 0.0, h: Optional[torch.Tensor] = None) -> None:
    """out_x[t] = table[id] * scale + bigram row + position row; ``bigram`` = (table, buckets, mul_prev, mul_cur) or None with
    ``previous`` int32 [slots, 1] the last token of every request slot; ``single``: every request brings one token.
    ``norm_w`` float32 [d]: the sum is RMS-normed with that weight; ``h`` (bf16) receives a copy of the result."""
    T, d = out_x.shape
    assert h is None or (h.dtype == torch.bfloat16 and h.is_contiguous() and h.shape == out_x.shape)
    assert out_x.dtype == torch.float32 and out_x.is_contiguous() and table.is_contiguous() and table.shape[1] == d
    bt, buckets, mp, mc = bigram if bigram is not None else (None, 0, 0, 0)
    assert bt is None or (bt.dtype == table.dtype and bt.is_contiguous() and tuple(bt.shape) == (buckets + 1, d))
    assert pos_table is None or (pos_table.dtype == table.dtype and pos_table.is_contiguous() and pos_table.shape[1] == d)
    _check(lib().infero_embed_compose(
        _ptr(table), c_int(_dt(table)), _ptr(_i32(ids, "ids")), _ptr(None if device_tokens is None else _i32(device_tokens, "device_tokens")),
        _ptr(out_x), c_int(T), c_int(d), c_int(table.shape[0]), c_float(scale), _ptr(bt), c_longlong(mp), c_longlong(mc),
        c_longlong(buckets), _ptr(None if previous is None else _i32(previous, "previous")), _ptr(_i32(tok_entry, "tok_entry")),
        _ptr(_i32(entry_q_start, "entry_q_start")), _ptr(_i32(entry_q_len, "entry_q_len")), _ptr(_i32(entry_slot, "entry_slot")),
        c_int(n_entries), _ptr(pos_table), c_int(pos_table.shape[0] if pos_table is not None else 0),
        _ptr(_i32(positions, "positions")), c_int(1 if single else 0), _ptr(_f32(norm_w, "norm_w")), c_float(eps), _ptr(h), _stream()))


# ---- recurrences with a matrix per head (csrc/outer_memory.cu) -------------------------------------------------------
MEMORY_RULES = {"delta": 0, "gated": 1}


def memory_tail_floats(taps: int, channels: int) -> int:
    """Floats of a convolution's tail in a memory's state slot (a multiple of four, so that what follows is aligned)."""
    return -(-(taps - 1) * channels // 4) * 4


def memory_state_floats(rule: str, heads: int, K: int, V: int, taps: int = 1, channels: int = 0) -> int:
    """Floats of one request's state: the convolution's last taps - 1 inputs, then S [heads, W, K] and, in the gated rule
    (W = V + 1), m [heads, W]; a multiple of four, so that every slot starts aligned."""
    W = V + 1 if rule == "gated" else V
    n = memory_tail_floats(taps, channels) + heads * W * K + (heads * W if rule == "gated" else 0)
    return -(-n // 4) * 4


def memory_prepare(proj: torch.Tensor, x_off: int, decay_off: int, step_off: int, conv_w: torch.Tensor, a_log: torch.Tensor,
                   dt_bias: torch.Tensor, state: torch.Tensor, tok_entry, entry_q_start, entry_q_len, entry_slot, n_entries: int,
                   G: int, H: int, K: int, V: int, single: bool):
    """From the 32-bit product rows ([q | k | v] at column ``x_off``, the raw decays and steps of the heads at theirs) to
    (u [T, 2 G K + H V], table [H, T, 12]): convolution over time (``conv_w`` float32 [taps, channels]) and silu, q and k unit
    vectors per head, q times K^-1/2; the gates, and the products of the scan's groups of four tokens (csrc/outer_memory.cu); the
    requests' tails (the first (taps - 1) channels numbers of their state) move on.  ``single``: every request of the step
    brings one token."""
    T = proj.shape[0]
    taps, CH = conv_w.shape
    assert CH == 2 * G * K + H * V and proj.dtype == torch.float32 and proj.stride(1) == 1
    assert proj.shape[1] >= max(x_off + CH, decay_off + H, step_off + H) and a_log.numel() == dt_bias.numel() == H
    assert state.dtype == torch.float32 and state.is_contiguous()
    u = torch.empty((T, CH), dtype=torch.float32, device=proj.device)
    table = torch.empty((H, T, 12), dtype=torch.float32, device=proj.device)
    L = lib()
    _check(L.infero_memory_prepare(_ptr(proj), c_longlong(proj.stride(0)), c_int(x_off), _ptr(_f32(conv_w, "conv_w")), c_int(taps),
                                   _ptr(state), c_longlong(state.stride(0)), _ptr(_i32(tok_entry, "tok_entry")),
                                   _ptr(_i32(entry_q_start, "entry_q_start")), _ptr(_i32(entry_slot, "entry_slot")), _ptr(u), _ptr(table),
                                   _ptr(_f32(a_log, "a_log")), _ptr(_f32(dt_bias, "dt_bias")), c_int(decay_off), c_int(step_off),
                                   c_int(T), c_int(G), c_int(H), c_int(K), c_int(V), c_int(1 if single else 0), _stream()))
    if not single:
        _check(L.infero_conv_tail(_ptr(proj[:, x_off:]), c_int(proj.stride(0)), c_int(taps), _ptr(state), c_longlong(state.stride(0)),
                                  _ptr(_i32(entry_q_start, "entry_q_start")), _ptr(_i32(entry_q_len, "entry_q_len")),
                                  _ptr(_i32(entry_slot, "entry_slot")), c_int(n_entries), c_int(CH), _stream()))
    return u, table


def memory_gates(gates: torch.Tensor, in_off: int, forget_off: int, cap: float, state: torch.Tensor, m_off: int, entry_q_start,
                 entry_q_len, entry_slot, n_entries: int, H: int, W: int) -> torch.Tensor:
    """The gated rule's gates of every token, [H, T, 4], from the raw ones; the requests' running maxima ([H, W] at ``m_off`` of
    their state) move on."""
    T = gates.shape[0]
    assert gates.dtype == torch.float32 and gates.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous()
    assert gates.shape[1] >= max(in_off, forget_off) + H and m_off + H * W <= state.shape[1]
    table = torch.empty((H, T, 4), dtype=torch.float32, device=gates.device)
    _check(lib().infero_memory_gates(_ptr(gates), c_longlong(gates.stride(0)), c_int(in_off), c_int(forget_off), c_float(cap), _ptr(state),
                                     c_longlong(state.stride(0)), c_longlong(m_off), _ptr(_i32(entry_q_start, "entry_q_start")),
                                     _ptr(_i32(entry_q_len, "entry_q_len")), _ptr(_i32(entry_slot, "entry_slot")), _ptr(table), c_int(T),
                                     c_int(n_entries), c_int(H), c_int(W), _stream()))
    return table


def _memory_scan(rule: str, src, q_off, k_off, v_off, table, gates, in_off, forget_off, cap, q_scale, state, s_off, entry_q_start,
                 entry_q_len, entry_slot, n_entries, H, G, K, V, single):
    from .tc_gemm import sm_count
    T = src.shape[0]
    gated = rule == "gated"
    assert src.dtype == torch.float32 and src.stride(1) == 1 and src.shape[1] >= max(q_off + G * K, k_off + G * K, v_off + H * V)
    assert state.dtype == torch.float32 and state.is_contiguous()
    assert s_off + H * (V + 1 if gated else V) * K + (H * (V + 1) if gated else 0) <= state.shape[1]
    y = torch.empty((T, H * V), dtype=torch.float32, device=src.device)
    den = torch.empty((T, H), dtype=torch.float32, device=src.device) if gated else None
    _check(lib().infero_memory_scan(
        c_int(MEMORY_RULES[rule]), _ptr(src), c_longlong(src.stride(0)), c_int(q_off), c_int(k_off), c_int(v_off), _ptr(table), c_int(T),
        _ptr(gates), c_longlong(gates.stride(0) if gates is not None else 0), c_int(in_off), c_int(forget_off), c_float(cap),
        c_float(q_scale), _ptr(state), c_longlong(state.stride(0)), c_longlong(s_off),
        _ptr(_i32(entry_q_start, "entry_q_start")), _ptr(_i32(entry_q_len, "entry_q_len")), _ptr(_i32(entry_slot, "entry_slot")),
        _ptr(y), _ptr(den), c_int(n_entries), c_int(1 if single else 0), c_int(H), c_int(G), c_int(K), c_int(V),
        c_int(sm_count(src.device)), _stream()))
    return y, den


def delta_scan(u: torch.Tensor, table: torch.Tensor, state: torch.Tensor, s_off: int, entry_q_start, entry_q_len, entry_slot,
               n_entries: int, H: int, G: int, K: int, V: int, single: bool = False) -> torch.Tensor:
    """The gated delta rule of every request over its new tokens, from what ``memory_prepare`` left (csrc/outer_memory.cu);
    float32 [T, H V], what the heads read out.  S [H, V, K] at ``s_off`` of the requests' state."""
    assert table.is_contiguous() and tuple(table.shape) == (H, u.shape[0], 12)
    return _memory_scan("delta", u, 0, G * K, 2 * G * K, table, None, 0, 0, 0.0, 1.0, state, s_off, entry_q_start, entry_q_len, entry_slot,
                        n_entries, H, G, K, V, single)[0]


def gated_scan(proj: torch.Tensor, q_off: int, k_off: int, v_off: int, in_off: int, forget_off: int, cap: float, state: torch.Tensor,
               s_off: int, entry_q_start, entry_q_len, entry_slot, n_entries: int, H: int, K: int, V: int, single: bool = False):
    """The matrix memory of every request over its new tokens, from the 32-bit product rows; (y float32 [T, H V], den float32
    [T, H]): what the heads read out, q times K^-1/2, and what it is yet to be divided by.  S and the normaliser [H, V + 1, K]
    at ``s_off`` of the requests' state, the running maximum [H, V + 1] behind it."""
    table = None
    if not single:
        table = memory_gates(proj, in_off, forget_off, cap, state, s_off + H * (V + 1) * K, entry_q_start, entry_q_len, entry_slot,
                             n_entries, H, V + 1)
    return _memory_scan("gated", proj, q_off, k_off, v_off, table, proj if single else None, in_off, forget_off, cap, K ** -0.5, state, s_off,
                        entry_q_start, entry_q_len, entry_slot, n_entries, H, H, K, V, single)


# ---- memories with a decay per channel of a key (csrc/low_rank.cu, channel_memory.cuh) -------------------------------
LOW_RANK_MODES = {"plain": 0, "decay": 1, "sigmoid": 2}


def low_rank(a: torch.Tensor, w: torch.Tensor, mode: str = "plain", bias: Optional[torch.Tensor] = None,
             a_log: Optional[torch.Tensor] = None, tau: float = 1.0, beside=None):
    """float32 [T, N] from a product's narrow middle ``a`` (float32 [T, R], a column slice) and w [N, R]: z = a w^T (+ bias);
    "decay": exp(-exp(a_log of the head) softplus(z)) with N / len(a_log) columns a head; "sigmoid": sigmoid(z)^(1 / tau).
    ``beside`` = (a2, w2): a second, plain product from columns of the same rows, in the same launch; both are returned then."""
    T, R = a.shape
    N = w.shape[0]
    assert a.dtype == torch.float32 and a.stride(1) == 1 and w.is_contiguous() and w.shape[1] == R
    assert bias is None or bias.numel() == N
    assert mode != "decay" or N % a_log.numel() == 0
    out = torch.empty((T, N), dtype=torch.float32, device=a.device)
    a2 = w2 = out2 = None
    if beside is not None:
        a2, w2 = beside
        assert a2.dtype == torch.float32 and a2.stride() == a.stride() and a2.shape[0] == T and w2.is_contiguous() and w2.shape[1] == a2.shape[1]
        out2 = torch.empty((T, w2.shape[0]), dtype=torch.float32, device=a.device)
    _check(lib().infero_low_rank(_ptr(a), c_longlong(a.stride(0)), _ptr(w), c_int(_dt(w)), _ptr(_f32(bias, "bias")), _ptr(_f32(a_log, "a_log")),
                                 c_int(N // a_log.numel() if a_log is not None else 1), c_float(tau), c_int(LOW_RANK_MODES[mode]), _ptr(out),
                                 c_int(T), c_int(N), c_int(R), _ptr(a2), _ptr(w2), c_int(_dt(w2) if w2 is not None else 0), _ptr(out2),
                                 c_int(w2.shape[0] if w2 is not None else 0), c_int(w2.shape[1] if w2 is not None else 0), _stream()))
    return out if out2 is None else (out, out2)


def decayed_records(a: torch.Tensor, w: torch.Tensor, bias: torch.Tensor, tau: float, proj: torch.Tensor, q_off: int, k_off: int, H: int,
                    K: int) -> torch.Tensor:
    """What the scan of gated linear attention reads: records [H, T, 3 Kp] of a token's decays sigmoid(a w^T + bias)^(1 / tau), its k
    and its q (columns of the 32-bit product rows ``proj``)."""
    T, R = a.shape
    assert a.dtype == proj.dtype == torch.float32 and a.stride(1) == proj.stride(1) == 1 and w.is_contiguous() and tuple(w.shape) == (H * K, R)
    assert bias.numel() == H * K and proj.shape[1] >= max(q_off, k_off) + H * K
    Kp = int(lib().infero_channel_rows(c_int(K)))
    rec = torch.empty((H, T, 3 * Kp), dtype=torch.float32, device=a.device)
    _check(lib().infero_low_rank_records(_ptr(a), c_longlong(a.stride(0)), _ptr(w), c_int(_dt(w)), _ptr(_f32(bias, "bias")), c_float(tau), _ptr(rec),
                                         c_int(Kp), _ptr(proj), c_longlong(proj.stride(0)), c_int(q_off), c_int(k_off), c_int(T), c_int(H),
                                         c_int(K), c_int(R), _stream()))
    return rec


def channel_prepare(proj: torch.Tensor, x_off: int, step_off: int, conv_w: torch.Tensor, decay: torch.Tensor, state: torch.Tensor,
                    tok_entry, entry_q_start, entry_q_len, entry_slot, n_entries: int, G: int, H: int, K: int, V: int, single: bool):
    """What the delta rule's scan needs where every channel of a key decays on its own: (values [T, H V], records [H, slots, n] of
    groups of four tokens) from the 32-bit product rows ([q | k | v] at ``x_off``, raw steps at ``step_off``) and the decays
    [T, H K]; see csrc/channel_memory.cuh.  The requests' tails (the convolution's last taps - 1 inputs) move on."""
    T = proj.shape[0]
    taps, CH = conv_w.shape
    assert CH == 2 * G * K + H * V and proj.dtype == torch.float32 and proj.stride(1) == 1 and proj.shape[1] >= max(x_off + CH, step_off + H)
    assert decay.dtype == torch.float32 and decay.is_contiguous() and tuple(decay.shape) == (T, H * K)
    assert state.dtype == torch.float32 and state.is_contiguous()
    L = lib()
    slots = int(L.infero_delta_slots(c_int(T), c_int(n_entries)))
    v = torch.empty((T, H * V), dtype=torch.float32, device=proj.device)
    rec = torch.empty((H, slots, int(L.infero_delta_record(c_int(K)))), dtype=torch.float32, device=proj.device)
    batch = (_ptr(_i32(entry_q_start, "entry_q_start")), _ptr(_i32(entry_q_len, "entry_q_len")), _ptr(_i32(entry_slot, "entry_slot")))
    _check(L.infero_channel_prepare(_ptr(proj), c_longlong(proj.stride(0)), c_int(x_off), _ptr(_f32(conv_w, "conv_w")), c_int(taps), _ptr(state),
                                    c_longlong(state.stride(0)), _ptr(_i32(tok_entry, "tok_entry")), *batch, _ptr(v), _ptr(rec), c_int(slots),
                                    _ptr(decay), c_int(step_off), c_int(T), c_int(G), c_int(H), c_int(K), c_int(V), c_int(1 if single else 0),
                                    _stream()))
    if not single:
        _check(L.infero_conv_tail(_ptr(proj[:, x_off:]), c_int(proj.stride(0)), c_int(taps), _ptr(state), c_longlong(state.stride(0)), *batch,
                                  c_int(n_entries), c_int(CH), _stream()))
    return v, rec


def _channel_scan(f, rec, n, v, extra, state, s_off, entry_q_start, entry_q_len, entry_slot, n_entries, H, K, V, single):
    from .tc_gemm import sm_count
    assert rec.is_contiguous() and rec.dtype == v.dtype == torch.float32 and v.stride(1) == 1 and v.shape[1] == H * V
    assert state.dtype == torch.float32 and state.is_contiguous() and s_off + H * V * K <= state.shape[1]
    y = torch.empty((v.shape[0], H * V), dtype=torch.float32, device=v.device)
    _check(f(_ptr(rec), c_int(n), _ptr(v), c_longlong(v.stride(0)), *extra, _ptr(state), c_longlong(state.stride(0)), c_longlong(s_off),
             _ptr(_i32(entry_q_start, "entry_q_start")), _ptr(_i32(entry_q_len, "entry_q_len")), _ptr(_i32(entry_slot, "entry_slot")), _ptr(y),
             c_int(n_entries), c_int(1 if single else 0), c_int(H), c_int(K), c_int(V), c_int(sm_count(v.device)), _stream()))
    return y


def channel_scan(v: torch.Tensor, rec: torch.Tensor, state: torch.Tensor, s_off: int, entry_q_start, entry_q_len, entry_slot,
                 n_entries: int, H: int, K: int, V: int, single: bool = False) -> torch.Tensor:
    """The delta rule with a decay per channel, from what ``channel_prepare`` left; float32 [T, H V].  S [H, V, K] at ``s_off``."""
    assert rec.shape[0] == H
    return _channel_scan(lib().infero_channel_scan, rec, rec.shape[1], v, (), state, s_off, entry_q_start, entry_q_len, entry_slot, n_entries,
                         H, K, V, single)


def decayed_scan(v: torch.Tensor, rec: torch.Tensor, state: torch.Tensor, s_off: int, entry_q_start, entry_q_len, entry_slot,
                 n_entries: int, H: int, K: int, V: int, single: bool = False) -> torch.Tensor:
    """Gated linear attention of every request over its new tokens, from the values (columns of the product's rows) and
    ``decayed_records``; float32 [T, H V], q times K^-1/2.  S [H, V, K] at ``s_off``."""
    assert tuple(rec.shape[:2]) == (H, v.shape[0])
    return _channel_scan(lib().infero_decayed_scan, rec, rec.shape[1], v, (c_float(K ** -0.5),), state, s_off, entry_q_start, entry_q_len,
                         entry_slot, n_entries, H, K, V, single)


def memory_finish(y: torch.Tensor, den: Optional[torch.Tensor], gate: torch.Tensor, act: str, norm_w: torch.Tensor, eps: float,
                  out: torch.Tensor, H: int, V: int, scale: float = 1.0) -> None:
    """out = (y / den) over its root mean square per head, times ``norm_w`` (V numbers shared by the heads, or H V), times
    ``act`` ("silu" or "sigmoid") of ``gate`` [T, H V], times ``scale``."""
    T = y.shape[0]
    assert y.is_contiguous() and tuple(y.shape) == (T, H * V) and gate.dtype == torch.float32 and gate.stride(1) == 1
    assert tuple(gate.shape) == (T, H * V) and out.shape == (T, H * V) and out.stride(1) == 1 and norm_w.numel() in (V, H * V)
    _check(lib().infero_memory_finish(_ptr(y), _ptr(den), _ptr(gate), c_int(gate.stride(0)), c_int({"sigmoid": 0, "silu": 1}[act]),
                                      _ptr(_f32(norm_w, "norm_w")), c_int(1 if norm_w.numel() == H * V else 0), c_float(eps),
                                      c_float(scale), _ptr(out), c_int(out.stride(0)), c_int(_dt(out)), c_int(T), c_int(H), c_int(V),
                                      _stream()))


def head_mix(a: torch.Tensor, mix: torch.Tensor, gate: Optional[torch.Tensor], out: torch.Tensor, H: int, G: int, V: int,
             scale: float = 1.0) -> None:
    """out[t, h] = (sum_g mix[h, g] a[t, h // (H / G), g]) * sigmoid(gate[t, h]) * scale, elementwise over V; a [T, G H V] as
    attention with ``cross`` leaves it; gate float32 [T, H V] or None; see csrc/head_mix.cu."""
    T = a.shape[0]
    assert tuple(a.shape) == (T, H * G * V) and a.stride(1) == 1 and tuple(out.shape) == (T, H * V) and out.stride(1) == 1
    assert tuple(mix.shape) == (H, H)
    assert gate is None or (gate.dtype == torch.float32 and tuple(gate.shape) == (T, H * V) and gate.stride(1) == 1)
    _check(lib().infero_head_mix(_ptr(a), c_int(a.stride(0)), c_int(_dt(a)), _ptr(_f32(mix, "mix")), _ptr(gate),
                                 c_int(gate.stride(0) if gate is not None else 0), _ptr(out), c_int(out.stride(0)), c_int(_dt(out)),
                                 c_int(T), c_int(H), c_int(G), c_int(V), c_float(scale), _stream()))


# ---- experts chosen by scores, ungated experts (csrc/moe.cu, csrc/moe_grouped.cu) -----------------------------------
def moe_select_scored(logits, E: int, top: int, renorm: bool = False):
    """From float32 logits [T, >= E] (a tensor, or ``Partials``: split-K sums that are added up here): scores
    sigmoid(logit); the ``top`` largest (lowest index wins a tie); (top_idx int32 [T, top], top_w float32 [T, top]) with
    top_w the chosen scores, over their sum where ``renorm``."""
    from . import Partials
    splits, split_stride = 1, 0
    if isinstance(logits, Partials):
        assert logits.bias is None
        splits, split_stride, logits = logits.splits, logits.split_stride, logits.data[0]
    T = logits.shape[0]
    assert logits.dtype == torch.float32 and logits.stride(1) == 1 and logits.shape[1] >= E
    idx = torch.empty((T, top), dtype=torch.int32, device=logits.device)
    w = torch.empty((T, top), dtype=torch.float32, device=logits.device)
    _check(lib().infero_moe_select_scored(_ptr(logits), c_int(logits.stride(0)), c_int(splits), c_longlong(split_stride),
                                          _ptr(idx), _ptr(w), c_int(T), c_int(E), c_int(top), c_int(1 if renorm else 0),
                                          _stream()))
    return idx, w


def moe_plain_streamed(h, up, down, top_idx, top_w, weight_input: bool, shared, y) -> None:
    """y[t] = sum_c expert_c(w_c h[t]) (``weight_input``) or sum_c w_c expert_c(h[t]), expert = down(relu(up x)^2),
    (+ shared[t]); every (token, choice) streams its expert's rows.  up [E, ff, d], down [E, d, ff].  ``shared``:
    float32 [T, d], or ``Partials`` of that shape (split-K sums, added up where they are used), or None."""
    from . import Partials
    sh_splits, sh_stride = 1, 0
    if isinstance(shared, Partials):
        assert shared.bias is None and tuple(shared.shape) == tuple(h.shape)
        sh_splits, sh_stride, shared = shared.splits, shared.split_stride, shared.data[0]
    T, d = h.shape
    E, ff, _ = up.shape
    top = top_idx.shape[1]
    assert up.dtype == h.dtype == down.dtype and up.is_contiguous() and down.is_contiguous() and h.stride(1) == 1
    assert tuple(down.shape) == (E, d, ff) and y.dtype == torch.float32 and y.is_contiguous() and y.shape == (T, d)
    scratch = torch.empty((T * top, ff), dtype=h.dtype, device=h.device)
    _check(lib().infero_moe_experts_plain_streamed(_ptr(h), c_int(h.stride(0)), _ptr(up), _ptr(down), c_int(_dt(h)),
                                                   _ptr(_i32(top_idx, "top_idx")), _ptr(_f32(top_w, "top_w")),
                                                   c_int(1 if weight_input else 0), _ptr(_f32(shared, "shared")),
                                                   c_int(sh_splits), c_longlong(sh_stride), _ptr(scratch), _ptr(y), c_int(T),
                                                   c_int(d), c_int(ff), c_int(top), _stream()))


def moe_plain_tc(h, up, down, top_idx, top_w, weight_input: bool, shared, y) -> None:
    """The same result by grouped products on the tcgen05 kernel (bf16): the tokens' rows are copied into expert order
    in tiles of 128 rows, times their pair's weight where it multiplies the expert's input; the first grouped product
    applies the squared relu in its epilogue; the rows of a token's choices are added up in ascending order."""
    from .tc_gemm import sm_count
    T, d = h.shape
    E, ff, _ = up.shape
    top = top_idx.shape[1]
    assert h.dtype == torch.bfloat16 and up.dtype == torch.bfloat16 and down.dtype == torch.bfloat16
    assert up.is_contiguous() and down.is_contiguous() and tuple(down.shape) == (E, d, ff)
    assert y.dtype == torch.float32 and y.is_contiguous() and y.shape == (T, d) and h.stride(1) == 1
    L = lib()
    tiles = int(L.infero_moe_tc_tiles(c_int(T * top), c_int(E)))
    R, dev = tiles * 128, h.device
    ints = torch.empty(2 * R + tiles + 1 + T * top, dtype=torch.int32, device=dev)
    sorted_pair, a_rows, tile_expert, pair_row = ints[:R], ints[R:2 * R], ints[2 * R:2 * R + tiles + 1], ints[2 * R + tiles + 1:]
    xs = torch.empty((R, d), dtype=torch.bfloat16, device=dev)
    _f32(top_w, "top_w")
    _check(L.infero_moe_tc_prepare_scaled(_ptr(h), c_int(h.stride(0)), _ptr(_i32(top_idx, "top_idx")), _ptr(sorted_pair),
                                          _ptr(a_rows), _ptr(tile_expert), _ptr(pair_row), _ptr(xs), c_int(T), c_int(d),
                                          c_int(E), c_int(top), _ptr(top_w if weight_input else None), _stream()))
    act = torch.empty((R, ff), dtype=torch.bfloat16, device=dev)
    sms = sm_count(dev)
    _check(L.infero_gemm_tc_grouped(_ptr(xs), _ptr(up), _ptr(act), c_int(2), c_int(R), c_int(ff), c_int(d), c_int(d),
                                    c_int(ff), _ptr(tile_expert), c_int(E), c_int(sms), *_act_args(None), _stream()))
    rows = torch.empty((R, d), dtype=torch.float32, device=dev)
    _check(L.infero_gemm_tc_grouped(_ptr(act), _ptr(down), _ptr(rows), c_int(0), c_int(R), c_int(d), c_int(ff), c_int(ff),
                                    c_int(d), _ptr(tile_expert), c_int(E), c_int(sms), *_act_args(None), _stream()))
    _check(L.infero_moe_tc_combine(_ptr(rows), _ptr(pair_row), _ptr(None if weight_input else top_w), _ptr(_f32(shared, "shared")),
                                   _ptr(None), _ptr(y), c_int(T), c_int(d), c_int(top), _stream()))
