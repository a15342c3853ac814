"""A plain, slow statement of the Dukolorn decoder on whole sequences, one function per mechanism, in 64-bit torch on the
CPU.  It is what the engine's kernels, cache and scheduler are held to; it shares nothing with the package.

Notation: h or x [T, d] is one sequence (positions 0..T-1); matrices are stored [out, in] and applied as y = x @ W.T; ``w``
maps tensor names to 64-bit tensors; ``cfg`` is the config.json dictionary; ``p`` the prefix of a mixer's tensors.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ---- small pieces ----------------------------------------------------------------------------------------------------
def unit_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def centred_norm(x, weight, eps):
    """An RMS norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1.0 + weight)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def causal_conv(x, taps_w):
    """x [T, C], taps_w [C, K] (the last column multiplies the current token), zeros before the sequence."""
    T, C = x.shape
    K = taps_w.shape[1]
    pad = torch.cat([torch.zeros(K - 1, C, dtype=x.dtype), x], dim=0)
    out = torch.zeros(T, C, dtype=x.dtype)
    for j in range(K):
        out = out + pad[j:j + T] * taps_w[:, j]
    return out


def low_rank(h, w, p: str, a: str, b: str):
    """A product through a narrow middle."""
    return (h @ w[f"{p}.{a}"].T) @ w[f"{p}.{b}"].T


def softmax_with_sink(s, sink):
    """Weights of scores s [H, T, T] (masked ones -inf) with one more term exp(sink[h]) in the denominator."""
    top = torch.maximum(s.amax(dim=-1), sink.view(-1, 1)).unsqueeze(-1)
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink.view(-1, 1, 1) - top))


# ---- mixer "parallel", left side: attention ------------------------------------------------------------------------------
def query_temperature(p: int, coef: float, every: float) -> float:
    """What a query at position p is multiplied by."""
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1)


def distance_bucket(n: int, B: int, D: float) -> int:
    half = B // 2
    if n < half:
        return n
    return min(B - 1, half + math.floor(math.log(n / half) / math.log(D / half) * (B - half)))


def soft_cap(s, cap: float):
    return cap * torch.tanh(s / cap)


def left_weights(h, w, p: str, m: dict, eps: float):
    """Softmax weights of every query head, [H, T, T]."""
    T = h.shape[0]
    H, G, K = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = (unit_rms(h @ w[p + ".q"].T, eps) * w[p + ".q.norm"]).view(T, H, K)
    k = (unit_rms(h @ w[p + ".k"].T, eps) * w[p + ".k.norm"]).view(T, G, K)
    if m.get("q_temp"):
        t = [query_temperature(i, float(m["q_temp"]["coef"]), float(m["q_temp"]["every"])) for i in range(T)]
        q = q * torch.tensor(t, dtype=q.dtype).view(T, 1, 1)
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, dim=1)) * float(m["scale"])
    if m.get("softcap"):
        s = soft_cap(s, float(m["softcap"]))
    rel = w[p + ".rel"]
    rows = [distance_bucket(n, rel.shape[0], float(m["bias_max"])) for n in range(T)]
    i, j = torch.arange(T).unsqueeze(1), torch.arange(T).unsqueeze(0)
    s = s + rel[torch.tensor(rows)][(i - j).clamp(min=0)].permute(2, 0, 1)
    return softmax_with_sink(s.masked_fill(j > i, float("-inf")), w[p + ".sink"])


def left_inner(h, w, p: str, m: dict, eps: float):
    """What the left mixer's output product takes, [T, heads * vdim]."""
    T = h.shape[0]
    H, G, V = int(m["heads"]), int(m["kv_heads"]), int(m["vdim"])
    v = (h @ w[p + ".v"].T).view(T, G, V).repeat_interleave(H // G, dim=1)
    return torch.einsum("hij,jhv->ihv", left_weights(h, w, p, m, eps), v).reshape(T, H * V)


# ---- mixer "parallel", right side: gated linear attention ----------------------------------------------------------------
def decayed_memory(q, k, v, alpha):
    """q (already scaled), k, alpha [T, H, K]; v [T, H, V].  S <- alpha S (alpha acts on the rows); S <- S + k v^T; o = S^T q."""
    T, H, K = q.shape
    S = torch.zeros(H, K, v.shape[2], dtype=q.dtype)
    outs = []
    for t in range(T):
        S = S * alpha[t].unsqueeze(2) + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        outs.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(outs)


def right_inner(h, w, p: str, m: dict, eps: float):
    T = h.shape[0]
    H, K, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + ".q"].T).view(T, H, K) * K ** -0.5
    k = (h @ w[p + ".k"].T).view(T, H, K)
    v = (h @ w[p + ".v"].T).view(T, H, V)
    z = low_rank(h, w, p, "a1", "a2") + w[p + ".a2.b"]
    alpha = (torch.sigmoid(z) ** (1.0 / float(m["tau"]))).view(T, H, K)
    o = unit_rms(decayed_memory(q, k, v, alpha), eps) * w[p + ".norm"]
    return o.reshape(T, H * V) * silu(h @ w[p + ".g"].T)


def parallel_mixer(h, w, p: str, m: dict, eps: float):
    left = left_inner(h, w, p + ".left", m["left"], eps) @ w[p + ".left.o"].T
    right = right_inner(h, w, p + ".right", m["right"], eps) @ w[p + ".right.o"].T
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


# ---- mixer "latent_attention" ------------------------------------------------------------------------------------------
def rotate_pairs(x, positions, dims: int, base: float):
    """x [T, ..., R]: of its first ``dims`` numbers every neighbouring pair turns by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(x.dtype) * base ** (-2.0 * i / dims)
        a = a.view(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def latent_inner(h, w, p: str, m: dict, eps: float):
    """What the latent mixer's output product takes, [T, heads * vdim]."""
    T = h.shape[0]
    H, D, R, V, C = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    pos = torch.arange(T)
    q = (h @ w[p + ".q"].T).view(T, H, D + R)
    kv = h @ w[p + ".dkv"].T
    c = unit_rms(kv[:, :C], eps) * w[p + ".dkv.norm"]
    dims, base = int(m["rot"]["dims"]), float(m["rot"]["base"])
    qr, kr = rotate_pairs(q[..., D:], pos, dims, base), rotate_pairs(kv[:, C:], pos, dims, base)
    k = (c @ w[p + ".uk"].T).view(T, H, D)
    v = (c @ w[p + ".uv"].T).view(T, H, V)
    s = (torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihr,jr->hij", qr, kr)) * float(m["scale"])
    i, j = pos.unsqueeze(1), pos.unsqueeze(0)
    hidden = j > i
    if m.get("mask"):
        hidden = hidden | (i - j >= int(m["mask"]["size"]))
    weights = softmax_with_sink(s.masked_fill(hidden, float("-inf")), w[p + ".sink"])
    return torch.einsum("hij,jhv->ihv", weights, v).reshape(T, H * V)


def latent_mixer(h, w, p: str, m: dict, eps: float):
    return latent_inner(h, w, p, m, eps) @ w[p + ".o"].T


# ---- mixer "channel_delta" ---------------------------------------------------------------------------------------------
def unit_vectors(x):
    return x / torch.sqrt(x.pow(2).sum(dim=-1, keepdim=True) + 1e-6)


def channel_delta_rule(q, k, v, beta, g):
    """q, k, g [T, H, K]; v [T, H, V]; beta [T, H].  Per head a memory S [K, V]:
    S <- g S (g acts on the rows);  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    T, H, K = q.shape
    S = torch.zeros(H, K, v.shape[2], dtype=q.dtype)
    outs = []
    for t in range(T):
        S = S * g[t].unsqueeze(2)
        u = beta[t].view(H, 1) * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t].unsqueeze(2) * u.unsqueeze(1)
        outs.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(outs)


def delta_inner(h, w, p: str, m: dict, eps: float):
    """What the delta mixer's output product takes, [T, heads * vdim]."""
    T = h.shape[0]
    H, G, K, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (silu(causal_conv(h @ w[f"{p}.{n}"].T, w[f"{p}.{n}.conv"])) for n in ("q", "k", "v"))
    q = unit_vectors(q.view(T, G, K)) * K ** -0.5
    k = unit_vectors(k.view(T, G, K))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ w[p + ".b"].T)
    steps = softplus(low_rank(h, w, p, "a1", "a2") + w[p + ".dt_bias"]).view(T, H, K)
    g = torch.exp(-torch.exp(w[p + ".A_log"]).view(1, H, 1) * steps)
    o = channel_delta_rule(q, k, v.view(T, H, V), beta, g)
    o = unit_rms(o, eps) * w[p + ".norm"]
    return o.reshape(T, H * V) * torch.sigmoid(low_rank(h, w, p, "g1", "g2"))


def delta_mixer(h, w, p: str, m: dict, eps: float):
    return delta_inner(h, w, p, m, eps) @ w[p + ".o"].T


# ---- feed-forward, layer, model ----------------------------------------------------------------------------------------
def biased_swiglu(h, w, p: str):
    lin = lambda x, n: x @ w[f"{p}.{n}"].T + w[f"{p}.{n}.b"]                     # noqa: E731
    return lin(silu(lin(h, "gate")) * lin(h, "up"), "down")


MIXERS = {"parallel": parallel_mixer, "latent_attention": latent_mixer, "channel_delta": delta_mixer}


def embed(cfg: dict, w, tokens: List[int]):
    return centred_norm(w["embed"][torch.tensor(tokens, dtype=torch.long)], w["embed.norm"], float(cfg["norm"]["eps"]))


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None):
    """Logits [T, vocab] of one sequence; ``residuals`` collects the residual stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = embed(cfg, w, tokens)
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}"
        x = x + centred_norm(MIXERS[L["type"]](x, w, p + ".mix", L["mixer"], eps), w[p + ".norm1"], eps)
        if L.get("mlp") is not None:
            x = x + centred_norm(biased_swiglu(x, w, p + ".mlp"), w[p + ".norm2"], eps)
        if residuals is not None:
            residuals.append(x.clone())
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T * float(cfg.get("logit_scale", 1.0))
