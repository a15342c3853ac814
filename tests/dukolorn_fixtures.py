"""Small Dukolorn configurations, random model folders and plain logits for the tests."""
from __future__ import annotations

import functools
import os
import random
import tempfile
from typing import Dict, List

import numpy as np
import torch

import plain_dukolorn as PD
import plain_qwen2

_TMP = tempfile.mkdtemp(prefix="infero_b200_dukolorn_")
# Largest |engine - plain| over a row of logits, relative to the request's largest |logit|: no row is above the first number,
# at most one in twenty above the second.  (A norm over a memory's read-out turns a read-out that happens to be near zero into
# a direction, which 16 bits do not hold: rounding nothing but the sublayers' inputs and results to bf16 in the plain
# statement moves single rows of these models by up to 0.22, half of the rows by less than 0.01.)
TOL = {"float32": (5e-4, 2e-5), "bfloat16": (0.4, 0.06)}


def delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def left(heads, kv, dim, vdim, scale, bias_max, softcap, temp):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max, "softcap": softcap,
            "q_temp": {"coef": temp[0], "every": temp[1]}}


def right(heads, dim, vdim, tau):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def latent(heads, dim, rot_dim, vdim, rank, scale, base, window):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
            "rot": {"base": base, "dims": rot_dim}, "mask": {"size": window}}


def par(l, r, ls, rs):
    return {"left": l, "right": r, "left_scale": ls, "right_scale": rs}


def _layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _config(vocab, width, eps, logit_scale, layers):
    return {"architecture": "Dukolorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


# A: sizes the tensor-core kernels take; grouped heads; a window that is no multiple of a page
A = _config(199, 128, 2e-5, 0.5, [
    _layer("parallel", par(left(4, 2, 64, 64, 0.11, 60, 6.0, (0.4, 32)), right(2, 32, 48, 8.0), 0.7, 1.4), 96),
    _layer("latent_attention", latent(4, 32, 16, 24, 64, 0.2, 5000.0, 39), 160),
    _layer("channel_delta", delta(4, 2, 64, 32, 3)),
    _layer("latent_attention", latent(2, 16, 32, 16, 128, 0.17, 900.0, 17))])
# B: odd sizes that no tensor-core kernel takes; values wider and narrower than keys; three kv heads; two taps; more
#    buckets than distances; narrow middles of one and three
B = _config(83, 36, 1e-6, 3.0, [
    _layer("channel_delta", delta(6, 3, 5, 10, 2), 20),
    _layer("latent_attention", latent(3, 6, 4, 5, 10, 0.4, 100.0, 7)),
    _layer("parallel", par(left(6, 3, 10, 6, 0.35, 12.5, 2.0, (0.9, 3)), right(3, 7, 9, 2.5), 1.7, 0.4)),
    _layer("parallel", par(left(2, 2, 6, 14, 0.4, 200, 30.0, (0.2, 7.5)), right(5, 18, 3, 30.0), 0.3, 2.0), 44)])
# C: values that make mechanisms vanish: one head everywhere, one tap, a window of one token, scales of 1, a temperature
#    that never moves, a root of 1, a bias that is the same at every distance but the last (two buckets)
C = _config(53, 40, 1e-5, 1.0, [
    _layer("latent_attention", latent(1, 8, 2, 8, 8, 0.3, 50.0, 1), 32),
    _layer("parallel", par(left(1, 1, 16, 16, 0.25, 2, 1000.0, (0.0, 1)), right(1, 8, 16, 1.0), 1.0, 1.0), 32),
    _layer("channel_delta", delta(1, 1, 8, 8, 1)),
    _layer("channel_delta", delta(3, 3, 20, 4, 5), 24)])
# D: heads of 128 for the bf16 kernels, keys of 128 rows in both memories, six taps
D = _config(257, 256, 1e-6, 0.8, [
    _layer("channel_delta", delta(4, 4, 128, 64, 6), 256),
    _layer("parallel", par(left(4, 2, 128, 128, 0.06, 150, 15.0, (0.25, 64)), right(2, 128, 128, 12.0), 1.3, 0.9), 256),
    _layer("latent_attention", latent(8, 64, 32, 32, 128, 0.1, 10000.0, 100), 256)])
# E: keys wider than values in the bf16 kernels' steps of 16, four kv heads; a window longer than any prompt; a large eps,
#    which counts in every norm; a cap that most scores reach
E = _config(131, 192, 5e-3, 2.0, [
    _layer("parallel", par(left(8, 4, 48, 16, 0.15, 90, 0.8, (1.5, 16)), right(6, 16, 40, 4.0), 2.0, 0.5), 128),
    _layer("latent_attention", latent(5, 24, 8, 40, 32, 0.25, 2000.0, 4000)),
    _layer("channel_delta", delta(8, 2, 24, 16, 4), 128)])
CONFIGS = {"A": A, "B": B, "C": C, "D": D, "E": E}
BUCKETS = {"A": 10, "B": 24, "C": 2, "D": 18, "E": 7}          # rows of the distance tables
RANKS = {"A": 12, "B": 3, "C": 1, "D": 40, "E": 33}            # widths of the narrow middles (the gate's: one more)


@functools.lru_cache(maxsize=None)
def model_dir(name: str, seed: int = 5, store: str = "bfloat16") -> str:
    """A random model folder.  Random projections give an almost flat softmax, which hides a wrong key, so the latent layers'
    query projections and the left mixers' query norms are made larger; random decays forget within a few tokens, which hides
    a lost state, so their biases are moved to where a state lasts for dozens of tokens; sinks and distance tables get entries
    of a unit and more, and the tensors whose sizes are the folder's own get the sizes above."""
    from safetensors.torch import load_file, save_file
    from infero_b200.loading import write_random_model_dir
    d = os.path.join(_TMP, f"{name}_{seed}_{store}")
    write_random_model_dir(d, CONFIGS[name], seed=seed, dtype=store, std=0.12, norm_std=0.15)
    p = os.path.join(d, "model.safetensors")
    w = load_file(p)
    g = torch.Generator().manual_seed(seed)
    for k in sorted(w):
        t = w[k].float()
        kind = CONFIGS[name]["layers"][int(k[1:k.index(".")])]["type"] if k[0] == "l" and k[1].isdigit() else ""
        leaf = k.rsplit(".", 1)[-1]
        if kind == "latent_attention" and k.endswith("mix.q"):
            t = t * 2.0
        if k.endswith("left.q.norm"):
            t = t * 2.5
        if leaf == "rel":
            t = torch.randn(BUCKETS[name], t.shape[1], generator=g) * 1.5
        if leaf == "sink":
            t = torch.randn(t.shape, generator=g) * 1.5
        rank = RANKS[name] + (1 if leaf in ("g1", "g2") else 0)
        if leaf in ("a1", "g1"):
            t = torch.randn(rank, t.shape[1], generator=g) * (2.0 / t.shape[1] ** 0.5)
        if leaf in ("a2", "g2"):
            t = torch.randn(t.shape[0], rank, generator=g) * (0.8 / rank ** 0.5)
        if leaf == "dt_bias":
            t = t - 3.5
        if k.endswith("a2.b"):
            t = t + 1.5
        w[k] = t.to(w[k].dtype).contiguous()
    save_file(w, p, metadata={"format": "pt"})
    return d


@functools.lru_cache(maxsize=None)
def plain_model(mdir: str):
    return plain_qwen2.read_model(mdir, torch.float64)


def plain_logits(mdir: str, reqs: Dict[str, List[int]]) -> Dict[str, np.ndarray]:
    cfg, w = plain_model(mdir)
    return {rid: PD.forward(cfg, w, toks).numpy() for rid, toks in reqs.items()}


def make_requests(name: str, lengths, seed: int = 0) -> Dict[str, List[int]]:
    rng = random.Random(seed)
    V = CONFIGS[name]["vocab"]
    return {f"r{i}": [rng.randrange(V) for _ in range(n)] for i, n in enumerate(lengths)}
