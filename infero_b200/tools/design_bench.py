"""Vufizen, Gositar or Banelix beside Qwen2, Pibavik beside Banelix, Nuvarax beside Pibavik and Banelix, or Dukolorn beside Nuvarax, at
equal layer sizes: whole prompt steps and decode steps, and the designs' own kernels one by one against their rooflines.

    python -m infero_b200.tools.design_bench [--design vufizen|gositar|banelix|pibavik|nuvarax|dukolorn] [--sizes s,m] [--prompt 2048]
                                             [--context 2048] [--batch 8] [--layers 8]

(also ``bench.py --designs``).  Random weights made on the device, bf16.  Per size two models of the same width
and depth: Vufizen (HGRN2 and differential-attention layers alternating, routed experts with a shared one) and
Qwen2 with the same head count, a head as wide as both maps together, and a feed-forward as wide as what one token
uses of the experts.  Steps are timed with CUDA events after warm-up, an L2 flush between timed steps; kernels are
timed alone the same way.  One JSON line at the end.

Gositar (``--design gositar``): latent attention in every layer (both mixer types alternating), dense squared-relu and
group-routed expert feed-forwards alternating, four residual streams; beside Qwen2 with the same head count, heads of
128, a quarter as many kv heads, and a feed-forward as wide as what one token uses on average.

Banelix (``--design banelix``): parallel layers (causal attention whose values are its keys beside a gated linear
recurrence) and windowed attention layers with a sink alternating, every second attention layer reading the keys and
values of the one before it; beside Qwen2 with the same width, head counts, heads of 128 and feed-forward.

Pibavik (``--design pibavik``): of every four layers one parallel layer (gated, normed window attention beside a state-space
recurrence), one window attention layer with a distance bias, one latent attention layer and one attention layer that reads
the keys and values of the one two before it, all with experts chosen by sigmoid scores and a shared expert; beside Banelix,
the closest of the other designs (parallel layers with a recurrence, window attention, borrowed caches), with the same width,
depth, head counts, window, recurrence width and a dense feed-forward as wide as what one token uses of the experts.

Nuvarax (``--design nuvarax``): delta-rule layers and parallel layers (attention with a learned distance bias and mixed heads
beside a gated matrix memory) alternating, a dense clamped gated feed-forward, norms before and after every sublayer and a
convolution on what every mixer reads; beside Pibavik (the closest mixers: biased attention, a recurrence with a matrix per
head) and Banelix (parallel layers with a dense feed-forward) of the same width, depth and (active) feed-forward width.

Dukolorn (``--design dukolorn``): of every four layers one delta-rule layer with decays per channel, two parallel layers (soft-capped
attention with a distance bias and learned sinks beside gated linear attention) and one latent attention layer over a window,
a dense SwiGLU with biases and a norm on every sublayer's result; beside Nuvarax (delta-rule memories, biased attention beside a
gated matrix memory) of the same width, depth, head counts, memory sizes and feed-forward.
"""
from __future__ import annotations

import argparse
import json
import os
import random
import sys
import types

SIZES = {
    "t": dict(width=256, heads=4, kv=2, dim=32, vdim=64, experts=4, top=2, ff=64, shared=128, vocab=1000),     # for tests
    "s": dict(width=1024, heads=8, kv=2, dim=64, vdim=128, experts=16, top=4, ff=512, shared=1024, vocab=32000),
    "m": dict(width=2048, heads=16, kv=4, dim=64, vdim=128, experts=32, top=4, ff=768, shared=1536, vocab=32000),
    "l": dict(width=4096, heads=32, kv=8, dim=64, vdim=128, experts=64, top=8, ff=768, shared=2048, vocab=32000),
}


GOSITAR_SIZES = {
    "t": dict(width=256, heads=4, dim=32, rot=16, vdim=32, rank=64, experts=4, top=2, groups=(2, 1), ff=64, shared=128, dense=512,
              streams=2, vocab=1000),                                                                         # for tests
    "s": dict(width=1024, heads=8, dim=64, rot=32, vdim=64, rank=256, experts=16, top=4, groups=(4, 2), ff=512, shared=1024,
              dense=4096, streams=4, vocab=32000),
    "m": dict(width=2048, heads=16, dim=128, rot=64, vdim=128, rank=512, experts=32, top=4, groups=(4, 2), ff=768, shared=1536,
              dense=6144, streams=4, vocab=32000),
    "l": dict(width=4096, heads=32, dim=128, rot=64, vdim=128, rank=512, experts=64, top=8, groups=(8, 4), ff=768, shared=2048,
              dense=8192, streams=4, vocab=32000),
}


def gositar_config(z, layers):
    mix = {"heads": z["heads"], "dim": z["dim"], "rot_dim": z["rot"], "vdim": z["vdim"], "kv_rank": z["rank"],
           "scale": (z["dim"] + z["rot"]) ** -0.5,
           "rot": {"base": 10000.0, "dims": z["rot"], "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    moe = {"kind": "moe", "expert": {"ff": z["ff"], "limit": 7.0}, "shared": {"ff": z["shared"], "limit": 7.0},
           "router": {"experts": z["experts"], "top": z["top"], "groups": {"count": z["groups"][0], "keep": z["groups"][1]}}}
    dense = {"kind": "dense", "ff": z["dense"]}
    return {"architecture": "Gositar", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5}, "streams": z["streams"],
            "layers": [{"type": "latent_attention" if i % 2 == 0 else "latent_attention_2", "mixer": mix,
                        "mlp": dense if i % 2 == 0 else moe} for i in range(layers)]}


def qwen2_beside_gositar(z, layers):
    used = (z["dense"] * 2 // 3 + z["top"] * z["ff"] + z["shared"]) // 2          # (two matrices of `dense` against three)
    return {"architectures": ["Qwen2ForCausalLM"], "model_type": "qwen2", "num_hidden_layers": layers,
            "hidden_size": z["width"], "num_attention_heads": z["heads"], "num_key_value_heads": max(1, z["heads"] // 4),
            "head_dim": 128, "intermediate_size": -(-used // 64) * 64, "vocab_size": z["vocab"],
            "rope_theta": 10000.0, "rms_norm_eps": 1e-5, "tie_word_embeddings": False}


BANELIX_SIZES = {
    "t": dict(width=256, heads=4, kv=2, dim=64, window=48, rec=256, blocks=4, taps=4, ff=512, vocab=1000),            # for tests
    "s": dict(width=1024, heads=8, kv=2, dim=128, window=1024, rec=1024, blocks=8, taps=4, ff=4096, vocab=32000),
    "m": dict(width=2048, heads=16, kv=4, dim=128, window=1024, rec=2048, blocks=16, taps=4, ff=6144, vocab=32000),
    "l": dict(width=4096, heads=32, kv=8, dim=128, window=1024, rec=4096, blocks=32, taps=4, ff=11008, vocab=32000),
}


PIBAVIK_SIZES = {
    "t": dict(width=256, heads=4, kv=2, dim=64, window=48, ssd_heads=8, ssd_vdim=32, state=32, groups=2, taps=4, norm_groups=2,
              kv_rank=64, q_rank=96, experts=4, top=2, ff=128, shared=256, vocab=1000),                          # for tests
    "s": dict(width=1024, heads=8, kv=2, dim=128, window=1024, ssd_heads=16, ssd_vdim=64, state=64, groups=2, taps=4, norm_groups=2,
              kv_rank=256, q_rank=512, experts=16, top=2, ff=1024, shared=2048, vocab=32000),
    "m": dict(width=2048, heads=16, kv=4, dim=128, window=1024, ssd_heads=32, ssd_vdim=64, state=128, groups=4, taps=4, norm_groups=4,
              kv_rank=512, q_rank=768, experts=32, top=2, ff=1536, shared=3072, vocab=32000),
    "l": dict(width=4096, heads=32, kv=8, dim=128, window=1024, ssd_heads=64, ssd_vdim=64, state=128, groups=8, taps=4, norm_groups=8,
              kv_rank=512, q_rank=1536, experts=64, top=4, ff=2048, shared=2816, vocab=32000),
}


NUVARAX_SIZES = {
    "t": dict(width=256, heads=4, kv=2, dim=64, bias_max=100, mem_heads=4, mem_dim=32, mem_vdim=64, delta_heads=4, delta_kv=2,
              delta_dim=32, delta_vdim=64, taps=4, ff=512, vocab=1000, beside="t"),                              # for tests
    "s": dict(width=1024, heads=4, kv=2, dim=128, bias_max=512, mem_heads=8, mem_dim=64, mem_vdim=128, delta_heads=8, delta_kv=4,
              delta_dim=64, delta_vdim=128, taps=4, ff=4096, vocab=32000, beside="s"),
    "m": dict(width=2048, heads=8, kv=2, dim=128, bias_max=512, mem_heads=16, mem_dim=128, mem_vdim=128, delta_heads=16, delta_kv=8,
              delta_dim=128, delta_vdim=128, taps=4, ff=6144, vocab=32000, beside="m"),
    "l": dict(width=4096, heads=16, kv=4, dim=128, bias_max=512, mem_heads=32, mem_dim=128, mem_vdim=128, delta_heads=32,
              delta_kv=16, delta_dim=128, delta_vdim=128, taps=4, ff=11008, vocab=32000, beside="l"),
}


DUKOLORN_SIZES = {
    "t": dict(NUVARAX_SIZES["t"], lat_heads=4, lat_dim=32, lat_rot=16, lat_vdim=32, lat_rank=64, window=48),      # for tests
    "s": dict(NUVARAX_SIZES["s"], lat_heads=8, lat_dim=64, lat_rot=32, lat_vdim=64, lat_rank=256, window=1024),
    "m": dict(NUVARAX_SIZES["m"], lat_heads=16, lat_dim=128, lat_rot=64, lat_vdim=128, lat_rank=512, window=1024),
    "l": dict(NUVARAX_SIZES["l"], lat_heads=32, lat_dim=128, lat_rot=64, lat_vdim=128, lat_rank=512, window=1024),
}


def dukolorn_config(z, layers):
    D = z["dim"]
    delta = {"heads": z["delta_heads"], "kv_heads": z["delta_kv"], "dim": z["delta_dim"], "vdim": z["delta_vdim"], "conv": z["taps"]}
    left = {"heads": z["heads"], "kv_heads": z["kv"], "dim": D, "vdim": D, "scale": D ** -0.5, "bias_max": z["bias_max"], "softcap": 30.0,
            "q_temp": {"coef": 0.1, "every": 1024}}
    par = {"left": left, "right": {"heads": z["mem_heads"], "dim": z["mem_dim"], "vdim": z["mem_vdim"], "tau": 16.0}, "left_scale": 0.9,
           "right_scale": 1.1}
    lat = {"heads": z["lat_heads"], "dim": z["lat_dim"], "rot_dim": z["lat_rot"], "vdim": z["lat_vdim"], "kv_rank": z["lat_rank"],
           "scale": (z["lat_dim"] + z["lat_rot"]) ** -0.5, "rot": {"base": 10000.0, "dims": z["lat_rot"]}, "mask": {"size": z["window"]}}
    kinds = [("channel_delta", delta), ("parallel", par), ("latent_attention", lat), ("parallel", par)]
    return {"architecture": "Dukolorn", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5}, "logit_scale": 0.5,
            "layers": [{"type": k, "mixer": m, "mlp": {"kind": "dense", "ff": z["ff"]}} for k, m in (kinds[i % 4] for i in range(layers))]}


def nuvarax_config(z, layers, max_positions=4096):
    D = z["dim"]
    delta = {"heads": z["delta_heads"], "kv_heads": z["delta_kv"], "dim": z["delta_dim"], "vdim": z["delta_vdim"], "conv": z["taps"]}
    left = {"heads": z["heads"], "kv_heads": z["kv"], "dim": D, "vdim": D, "scale": D ** -0.5, "bias_max": z["bias_max"]}
    right = {"heads": z["mem_heads"], "dim": z["mem_dim"], "vdim": z["mem_vdim"], "gate_cap": 15.0}
    mlp = {"kind": "dense", "ff": z["ff"], "limit": 7.0}
    return {"architecture": "Nuvarax", "vocab": z["vocab"], "width": z["width"], "max_positions": max_positions, "norm": {"eps": 1e-5},
            "embedding": {"scale": 1.0, "bigram": {"buckets": 2 * z["vocab"] + 1, "mul_prev": 31, "mul_cur": 17}}, "canon": {"taps": 4},
            "layers": [{"type": "delta", "mixer": delta, "mlp": mlp} if i % 2 == 0 else
                       {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp} for i in range(layers)]}


def pibavik_config(z, layers):
    D = z["dim"]
    left = {"heads": max(1, z["heads"] // 2), "kv_heads": max(1, z["kv"] // 2), "dim": D, "vdim": D, "scale": D ** -0.5,
            "mask": {"size": z["window"]}, "rot": {"base": 500000.0, "dims": D // 2}}
    right = {"heads": z["ssd_heads"], "vdim": z["ssd_vdim"], "state": z["state"], "groups": z["groups"], "conv": z["taps"],
             "norm_groups": z["norm_groups"]}
    par = {"left": left, "right": right, "left_scale": 0.7, "right_scale": 0.7}
    att = {"heads": z["heads"], "kv_heads": z["kv"], "dim": D, "vdim": D, "scale": D ** -0.5, "mask": {"size": z["window"]}}
    lat = {"heads": z["heads"], "dim": D, "vdim": D, "kv_rank": z["kv_rank"], "q_rank": z["q_rank"], "scale": D ** -0.5}
    mlp = {"kind": "moe", "expert": {"ff": z["ff"]}, "router": {"experts": z["experts"], "top": z["top"]}, "shared": {"ff": z["shared"]}}
    out = []
    for i in range(layers):
        if i % 4 == 0:
            out.append({"type": "parallel", "mixer": par, "mlp": mlp})
        elif i % 4 == 2:
            out.append({"type": "latent_attention", "mixer": lat, "mlp": mlp})
        else:
            out.append({"type": "attention", "mixer": dict(att, kv_from=i - 2) if i % 4 == 3 else att, "mlp": mlp})
    return {"architecture": "Pibavik", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
            "layers": out}


def banelix_beside_pibavik(z, layers):
    b = dict(width=z["width"], heads=z["heads"], kv=z["kv"], dim=z["dim"], window=z["window"], rec=z["ssd_heads"] * z["ssd_vdim"],
             blocks=z["heads"], taps=z["taps"], ff=z["top"] * z["ff"] + z["shared"], vocab=z["vocab"])
    return banelix_config(b, layers)


def banelix_config(z, layers):
    D = z["dim"]
    left = {"heads": max(1, z["heads"] // 2), "kv_heads": max(1, z["kv"] // 2), "dim": D, "vdim": D, "scale": D ** -0.5,
            "rot": {"base": 500000.0, "dims": D // 2, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    par = {"left": left, "right": {"width": z["rec"], "blocks": z["blocks"], "conv": z["taps"]}, "left_scale": 0.7, "right_scale": 0.7}
    att = {"heads": z["heads"], "kv_heads": z["kv"], "dim": D, "vdim": D, "scale": D ** -0.5, "mask": {"size": z["window"]},
           "rot": {"base": 10000.0, "dims": D, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    mlp = {"kind": "dense", "ff": z["ff"]}
    out = []
    for i in range(layers):
        if i % 2 == 0:
            out.append({"type": "parallel", "mixer": par, "mlp": mlp})
        else:
            out.append({"type": "attention", "mixer": dict(att, kv_from=i - 2) if i % 4 == 3 else att, "mlp": mlp})
    return {"architecture": "Banelix", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
            "residual_mult": 0.5, "layers": out}


def qwen2_beside_banelix(z, layers):
    return {"architectures": ["Qwen2ForCausalLM"], "model_type": "qwen2", "num_hidden_layers": layers,
            "hidden_size": z["width"], "num_attention_heads": z["heads"], "num_key_value_heads": z["kv"],
            "head_dim": z["dim"], "intermediate_size": z["ff"], "vocab_size": z["vocab"],
            "rope_theta": 10000.0, "rms_norm_eps": 1e-5, "tie_word_embeddings": False}


def vufizen_config(z, layers):
    mlp = {"kind": "moe", "router": {"experts": z["experts"], "top": z["top"]}, "expert": {"ff": z["ff"]},
           "shared": {"ff": z["shared"]}}
    att = {"heads": z["heads"], "kv_heads": z["kv"], "dim": z["dim"], "vdim": z["vdim"], "conv": 4, "diff": 0.5,
           "rot": {"base": 10000.0, "dims": z["dim"]}, "scale": z["dim"] ** -0.5}
    hg = {"heads": z["heads"], "dim": z["dim"], "vdim": z["vdim"]}
    return {"architecture": "Vufizen", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5},
            "layers": [{"type": "hgrn2" if i % 2 == 0 else "attention", "mixer": hg if i % 2 == 0 else att, "mlp": mlp}
                       for i in range(layers)]}


def qwen2_config(z, layers):
    return {"architectures": ["Qwen2ForCausalLM"], "model_type": "qwen2", "num_hidden_layers": layers,
            "hidden_size": z["width"], "num_attention_heads": z["heads"], "num_key_value_heads": z["kv"],
            "head_dim": 2 * z["dim"], "intermediate_size": z["top"] * z["ff"] + z["shared"], "vocab_size": z["vocab"],
            "rope_theta": 10000.0, "rms_norm_eps": 1e-5, "tie_word_embeddings": False}


class _Timer:
    def __init__(self):
        import torch
        self.torch = torch
        self.flush = torch.empty(192 << 20, dtype=torch.uint8, device="cuda")

    def __call__(self, fn, reps=7, warmup=3, setup=None):
        torch = self.torch
        if setup is None:
            # a kernel alone: replayed from a captured graph, so that the host's share of a launch is not timed
            fn()
            torch.cuda.synchronize()
            try:
                graph = torch.cuda.CUDAGraph()
                with torch.cuda.graph(graph):
                    from infero_b200 import kernels as K
                    with K.stream_scope():
                        fn()
                fn = graph.replay
            except Exception:                          # noqa: BLE001  (something in fn cannot be captured: time it as it is)
                torch.cuda.synchronize()
        times = []
        for i in range(warmup + reps):
            if setup:
                setup()
            self.flush.fill_(i & 255)
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            if i >= warmup:
                times.append(e0.elapsed_time(e1))
        times.sort()
        return times[len(times) // 2]


def time_model(cfg, prompt, context, batch, timer):
    import torch
    from infero_b200.config import EngineConfig
    from infero_b200.engine import ModelRunner, StepEntry
    from infero_b200.loading import random_model
    model, _ = random_model(cfg, seed=0, dtype="bfloat16", device="cuda:0", generate_on_device=True)
    vocab = model.spec.vocab_size
    rng = random.Random(1)
    ps = 16
    toks = lambda n: [rng.randrange(vocab) for _ in range(n)]                   # noqa: E731
    runner = ModelRunner(model, EngineConfig(dtype="bfloat16", page_size=ps, num_pages=2 * (-(-prompt // ps)), max_seqs=2,
                                             ctx=prompt, max_batch_tokens=prompt, cuda_graphs=False))
    p = toks(prompt)

    def prefill():
        runner.step([StepEntry("p", p, [prompt - 1])])
    pre_ms = timer(prefill, setup=lambda: (("p" in runner.manager.requests) and runner.close("p"), runner.open("p")))
    del runner
    torch.cuda.empty_cache()
    steps = 24
    runner = ModelRunner(model, EngineConfig(dtype="bfloat16", page_size=ps, num_pages=batch * (-(-(context + 64) // ps)),
                                             max_seqs=batch, ctx=context + 64, max_batch_tokens=max(2048, batch),
                                             max_logit_rows=max(8, batch), cuda_graphs=True))
    rids = [f"d{i}" for i in range(batch)]
    for r in rids:
        runner.open(r)
        done = 0
        while done < context - steps:
            n = min(2048, context - steps - done)
            runner.step([StepEntry(r, toks(n), [])])
            done += n
    for _ in range(4):                                     # eager, captured, replayed
        runner.step([StepEntry(r, toks(1), [0]) for r in rids])
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(steps - 4):
        runner.step([StepEntry(r, toks(1), [0]) for r in rids])
    e1.record()
    torch.cuda.synchronize()
    dec_ms = e0.elapsed_time(e1) / (steps - 4)
    out = {"prefill_tok_s": round(prompt / pre_ms * 1e3, 1), "prefill_ms": round(pre_ms, 3),
           "decode_tok_s": round(batch / dec_ms * 1e3, 1), "decode_ms_per_step": round(dec_ms, 4),
           "weight_mib": model.weight_bytes() >> 20, "graph_replays": runner.graph_replays}
    del runner, model
    torch.cuda.empty_cache()
    return out


def time_kernels(z, T, context, batch, timer, peaks):
    """The new design's kernels alone, each beside the kernel of the built-in decoder that does the like job."""
    import numpy as np
    import torch
    from infero_b200 import kernels as K
    from infero_b200.kernels import attention as A, diff_attention as DA, layer_ops as L, moe as M, tc_gemm
    from infero_b200.parts.linear import Linear
    dev, bf = "cuda:0", torch.bfloat16
    d, H, G, D, V = z["width"], z["heads"], z["kv"], z["dim"], z["vdim"]
    E, top, ff = z["experts"], z["top"], z["ff"]
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf, k=1.0: (torch.randn(s, generator=g, device=dev) * k).to(dtype)     # noqa: E731
    i32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.int32, device=dev)                 # noqa: E731
    hbm, tfl = peaks["hbm_gbs"], peaks["bf16_tflops"]
    rows = {}

    def note(name, ms, bytes_=0.0, flops=0.0):
        r = {"us": round(ms * 1e3, 1)}
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["hbm_frac"] = round(bytes_ / ms / 1e6 / hbm, 3)
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 1)
            r["tensor_frac"] = round(flops / ms / 1e9 / tfl, 3)
        rows[name] = r

    def batch_ctx(q_lens, pos0, ps=16):
        E_ = len(q_lens)
        per = [-(-(p + n) // ps) for p, n in zip(pos0, q_lens)]
        table = torch.full((E_, max(per)), -1, dtype=torch.int32)
        at = 0
        for e, n in enumerate(per):
            table[e, :n] = torch.arange(at, at + n, dtype=torch.int32)
            at += n
        qs = np.concatenate([[0], np.cumsum(q_lens)[:-1]])
        ctx = types.SimpleNamespace(
            n_entries=E_, n_tokens=int(sum(q_lens)), h_q_len=np.asarray(q_lens, dtype=np.int32), h_pos0=np.asarray(pos0, dtype=np.int32),
            tok_entry=i32(np.repeat(np.arange(E_), q_lens)), positions=i32(np.concatenate([p + np.arange(n) for p, n in zip(pos0, q_lens)])),
            entry_q_start=i32(qs), entry_q_len=i32(q_lens), entry_pos0=i32(pos0), entry_slot=i32(np.arange(E_)), kv_bound=None)
        return ctx, table.to(dev), at

    # ---- attention: prompt of T tokens, then `batch` single tokens at `context` -----------------------------------
    for label, q_lens, pos0 in (("prefill", [T], [0]), ("decode", [1] * batch, [context - 1] * batch)):
        ctx, table, pages = batch_ctx(q_lens, pos0)
        n = ctx.n_tokens
        kd, vd = rnd(pages, G, 16, 2 * D), rnd(pages, G, 16, V)
        kv = types.SimpleNamespace(k=kd, v=vd, page_size=16)
        padded = DA.as_plain_heads(bf, D, V, 16)
        q, out = rnd(n, 2 * H * D * (2 if padded else 1)), torch.empty(n, H * V, dtype=bf, device=dev)
        keys = sum(p + (n_ + 1) / 2 * 1 for p, n_ in zip(pos0, q_lens)) if label == "decode" else T / 2
        fl = 2.0 * H * (2 * D + 2 * V) * (T * T / 2 if label == "prefill" else batch * context)
        by = 2.0 * G * (2 * D + V) * (T if label == "prefill" else batch * context) + 2.0 * n * (2 * H * D + H * V)
        ms = timer(lambda: DA.paged_diff_attention(ctx, q, out, kv, table, H, G, D, V, None, D ** -0.5, 0.4, 1e-5, 0.5, q_padded=padded))
        note(f"diff_attention_{label}", ms, by, fl)
        # the built-in attention with a head as wide as both maps (2 D) and values of the same width
        Dq = 2 * D
        k2, v2 = rnd(pages, G, 16, Dq), rnd(pages, G, 16, Dq)
        q2, out2 = rnd(n, H * Dq), torch.empty(n, H * Dq, dtype=bf, device=dev)
        fl2 = 2.0 * H * 2 * Dq * (T * T / 2 if label == "prefill" else batch * context)
        by2 = 2.0 * G * 2 * Dq * (T if label == "prefill" else batch * context) + 4.0 * n * H * Dq
        ms = timer(lambda: A.attention_any(q2, out2, k2, v2, table, ctx.tok_entry, ctx.positions, H, G, Dq, 16, None, Dq ** -0.5,
                                           ctx.h_q_len, ctx.h_pos0, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_pos0))
        note(f"gqa_attention_{label}", ms, by2, fl2)
        if label == "prefill":      # the built-in kernel on the warp-level tensor cores (what head sizes other than 64 and 128 get)
            ms = timer(lambda: A.prefill(q2, out2, k2, v2, table, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_pos0, 1, 0,
                                         -(-T // 64), H, G, Dq, 16, None, Dq ** -0.5))
            note("gqa_attention_prefill_mma_sync", ms, by2, fl2)

    # ---- the recurrence ------------------------------------------------------------------------------------------
    for label, q_lens in (("prefill", [T]), ("decode", [1] * batch)):
        ctx, _, _ = batch_ctx(q_lens, [0] * len(q_lens))
        n = ctx.n_tokens
        proj = rnd(n, 2 * H * D + H * V, dtype=torch.float32)
        state = torch.zeros(len(q_lens), H, D, V, device=dev)
        fb, lo, wn = rnd(H * D, dtype=torch.float32), torch.rand(H * D, device=dev), torch.ones(V, device=dev)
        out = torch.empty(n, H * V, dtype=bf, device=dev)
        ms = timer(lambda: L.hgrn2_scan(proj, 0, H * D, 2 * H * D, fb, lo, wn, 1e-5, state, ctx.entry_q_start, ctx.entry_q_len,
                                        ctx.entry_slot, out, len(q_lens), H, D, V, q_lens=q_lens))
        note(f"hgrn2_scan_{label}", ms, 4.0 * n * (2 * H * D + H * V) + 2.0 * n * H * V + 8.0 * len(q_lens) * H * D * V)

    # ---- feed-forward: routed experts beside a dense SwiGLU of the width one token uses -----------------------------
    gu, dn = rnd(E, 2 * ff, d, k=0.05), rnd(E, d, ff, k=0.05)
    router = rnd(E, d, k=0.1)
    dense_ff = top * ff
    wgu, wdn = rnd(2 * dense_ff, d, k=0.05), rnd(d, dense_ff, k=0.05)
    for label, n in (("prefill", T), ("decode", batch)):
        h = rnd(n, d)
        y = torch.empty(n, d, device=dev)
        route = Linear(router)
        idx, w, _ = L.moe_select(route.forward(h, out_dtype=torch.float32), E, top)
        ms = timer(lambda: L.moe_select(route.forward(h, out_dtype=torch.float32), E, top))
        note(f"moe_route_{label}", ms, 2.0 * (n * d + E * d))
        used = min(E, n * top)
        ms = timer(lambda: M.experts(h, gu, dn, idx, w, None, None, y))
        note(f"moe_experts_{label}", ms, 2.0 * used * 3 * ff * d + 2.0 * n * d + 4.0 * n * d, 6.0 * n * top * ff * d)
        act = torch.empty(n, dense_ff, dtype=bf, device=dev)
        o = torch.empty(n, d, dtype=torch.float32, device=dev)

        def dense():
            if not tc_gemm.gemm_swiglu(h, wgu, act):
                K.swiglu(K.Partials(tc_gemm.partials(h, wgu)), act)
            tc_gemm.gemm(act, wdn, None, o)
        ms = timer(dense)
        note(f"dense_swiglu_{label}", ms, 2.0 * 3 * dense_ff * d + 6.0 * n * d, 6.0 * n * dense_ff * d)

    # ---- the small kernels -----------------------------------------------------------------------------------------
    x, yv, gl = rnd(T, d, dtype=torch.float32), rnd(T, d, dtype=torch.float32), rnd(T, d, dtype=torch.float32)
    gb, nw, hb = rnd(d, dtype=torch.float32), torch.ones(1, device=dev), torch.empty(T, d, dtype=bf, device=dev)
    ms = timer(lambda: L.gated_scalar_norm_add(x, yv, gl, gb, nw, 1e-5, hb))
    note("gated_norm_add_prefill", ms, T * d * (4 + 4 + 4 + 4 + 2))
    wv = torch.ones(d, device=dev)
    ms = timer(lambda: K.add_rmsnorm(x, yv, wv, 1e-5, hb))
    note("add_rmsnorm_prefill", ms, T * d * (4 + 4 + 4 + 2))
    ctx, table, pages = batch_ctx([T], [0])
    C = 2 * H * D + 2 * G * D + G * V
    proj, cw = rnd(T, C, dtype=torch.float32), rnd(4, C, dtype=torch.float32)
    st = torch.zeros(1, 3, C, device=dev)
    kd, vd = torch.empty(pages, G, 16, 2 * D, dtype=bf, device=dev), torch.empty(pages, G, 16, V, dtype=bf, device=dev)
    qn, inv = torch.ones(D, device=dev), torch.rand(D // 2, device=dev)
    qo = torch.empty(T, 2 * H * D, dtype=bf, device=dev)
    ms = timer(lambda: L.qkv_prepare(proj, cw, 4, st, qn, qn, 1e-5, inv, ctx.positions, ctx.tok_entry, ctx.entry_q_start,
                                     ctx.entry_slot, table, qo, kd, vd, 16, 2 * H, 2 * G, G, D, V))
    note("qkv_prepare_prefill", ms, T * C * (4 + 2))
    Dq = 2 * D
    qkv = rnd(T, (H + 2 * G) * Dq)
    k2, v2 = torch.empty(pages, G, 16, Dq, dtype=bf, device=dev), torch.empty(pages, G, 16, Dq, dtype=bf, device=dev)
    inv2 = torch.rand(Dq // 2, device=dev)
    ms = timer(lambda: K.rope_cache(qkv, ctx.positions, ctx.tok_entry, table, inv2, k2, v2, H, G, Dq, 16))
    note("rope_cache_prefill", ms, T * (H + 2 * G) * Dq * 2 * 2)
    return rows


def time_gositar_kernels(z, T, context, batch, timer, peaks):
    """Gositar's kernels alone, each beside the kernel of the built-in decoder that does the like job."""
    import numpy as np
    import torch
    from infero_b200 import kernels as K
    from infero_b200.kernels import attention as A, latent_attention as LA, layer_ops as L, moe as M, tc_gemm
    from infero_b200.parts.linear import Linear
    dev, bf = "cuda:0", torch.bfloat16
    d, H, D, R, V, C, S = z["width"], z["heads"], z["dim"], z["rot"], z["vdim"], z["rank"], z["streams"]
    E, top, ff = z["experts"], z["top"], z["ff"]
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf, k=1.0: (torch.randn(s, generator=g, device=dev) * k).to(dtype)     # noqa: E731
    i32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.int32, device=dev)                 # noqa: E731
    hbm, tfl = peaks["hbm_gbs"], peaks["bf16_tflops"]
    rows = {}

    def note(name, ms, bytes_=0.0, flops=0.0):
        r = {"us": round(ms * 1e3, 1)}
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["hbm_frac"] = round(bytes_ / ms / 1e6 / hbm, 3)
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 1)
            r["tensor_frac"] = round(flops / ms / 1e9 / tfl, 3)
        rows[name] = r

    def batch_ctx(q_lens, pos0, ps=16):
        E_ = len(q_lens)
        per = [-(-(p + n) // ps) for p, n in zip(pos0, q_lens)]
        table = torch.full((E_, max(per)), -1, dtype=torch.int32)
        at = 0
        for e, n in enumerate(per):
            table[e, :n] = torch.arange(at, at + n, dtype=torch.int32)
            at += n
        qs = np.concatenate([[0], np.cumsum(q_lens)[:-1]])
        ctx = types.SimpleNamespace(
            n_entries=E_, n_tokens=int(sum(q_lens)), h_q_len=np.asarray(q_lens, dtype=np.int32), h_pos0=np.asarray(pos0, dtype=np.int32),
            tok_entry=i32(np.repeat(np.arange(E_), q_lens)), positions=i32(np.concatenate([p + np.arange(n) for p, n in zip(pos0, q_lens)])),
            entry_q_start=i32(qs), entry_q_len=i32(q_lens), entry_pos0=i32(pos0), entry_slot=i32(np.arange(E_)), kv_bound=None)
        return ctx, table.to(dev), at

    G, Dq = max(1, H // 4), 128
    for label, q_lens, pos0 in (("prefill", [T], [0]), ("decode", [1] * batch, [context - 1] * batch)):
        ctx, table, pages = batch_ctx(q_lens, pos0)
        n = ctx.n_tokens
        pairs = T * T / 2 if label == "prefill" else batch * context           # (query, key) pairs per head
        keys = T if label == "prefill" else batch * context
        # ---- attention over the latent rows ------------------------------------------------------------------------
        kv = types.SimpleNamespace(k=rnd(pages, 1, 16, C + R), v=None, page_size=16, group=0)
        rows_h = -(-n // 128) * 128
        q_lat, q_rot = rnd(H, rows_h, C, dtype=torch.float32), rnd(H, rows_h, R, dtype=torch.float32)
        o_lat = torch.empty(H, rows_h, C, dtype=bf, device=dev)
        ms = timer(lambda: LA.attention(ctx, q_lat, q_rot, o_lat, kv, table, n, H, C, R, (D + R) ** -0.5))
        note(f"latent_attention_{label}", ms, 2.0 * (C + R) * keys + n * H * (4.0 * (C + R) + 2.0 * C), 2.0 * H * (2 * C + R) * pairs)
        rows[f"latent_attention_{label}"]["unabsorbed_tflops"] = round(2.0 * H * (D + R + V) * pairs / ms / 1e9, 1)
        # ---- the per-head products around it -----------------------------------------------------------------------
        q_plain, up_k = rnd(H, rows_h, D), rnd(H, C, D, k=0.05)
        ms = timer(lambda: LA.per_head_product(q_plain, up_k, q_lat, n))
        note(f"per_head_up_k_{label}", ms, 2.0 * H * C * D + H * rows_h * (2.0 * D + 4.0 * C), 2.0 * H * rows_h * C * D)
        up_v, val = rnd(H, V, C, k=0.05), torch.empty(H, rows_h, V, dtype=torch.float32, device=dev)
        ms = timer(lambda: LA.per_head_product(o_lat, up_v, val, n))
        note(f"per_head_up_v_{label}", ms, 2.0 * H * C * V + H * rows_h * (2.0 * C + 4.0 * V), 2.0 * H * rows_h * C * V)
        # ---- prepare beside rotary + cache append --------------------------------------------------------------------
        width = H * (D + R) + C + R + H
        proj, nw, fr = rnd(n, width, dtype=torch.float32), torch.ones(C, device=dev), torch.rand(R // 2, device=dev, dtype=torch.float64)
        ms = timer(lambda: LA.prepare(proj, 0, H * (D + R), nw, 1e-5, fr, "adjacent", 1.2, ctx.positions, ctx.tok_entry, table, kv.k,
                                      16, q_plain, q_rot, n, H, D, R, C))
        note(f"latent_prepare_{label}", ms, n * (4.0 * width + 2.0 * (C + R) + H * (2.0 * D + 4.0 * R)))
        gate, attn = proj[:, width - H:], torch.empty(n, H * V, dtype=bf, device=dev)
        ms = timer(lambda: LA.finish(val, gate, attn, n, H, V))
        note(f"latent_finish_{label}", ms, n * H * V * 6.0)
        # ---- the built-in attention: heads of 128, a quarter as many kv heads ----------------------------------------
        k2, v2 = rnd(pages, G, 16, Dq), rnd(pages, G, 16, Dq)
        q2, out2 = rnd(n, H * Dq), torch.empty(n, H * Dq, dtype=bf, device=dev)
        ms = timer(lambda: A.attention_any(q2, out2, k2, v2, table, ctx.tok_entry, ctx.positions, H, G, Dq, 16, None, Dq ** -0.5,
                                           ctx.h_q_len, ctx.h_pos0, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_pos0))
        note(f"gqa_attention_{label}", ms, 2.0 * G * 2 * Dq * keys + 4.0 * n * H * Dq, 2.0 * H * 2 * Dq * pairs)
        if label == "prefill":
            ms = timer(lambda: A.prefill(q2, out2, k2, v2, table, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_pos0, 1, 0,
                                         -(-T // 64), H, G, Dq, 16, None, Dq ** -0.5))
            note("gqa_attention_prefill_mma_sync", ms, 2.0 * G * 2 * Dq * keys + 4.0 * n * H * Dq, 2.0 * H * 2 * Dq * pairs)
        qkv = rnd(n, (H + 2 * G) * Dq)
        inv2 = torch.rand(Dq // 2, device=dev)
        ms = timer(lambda: K.rope_cache(qkv, ctx.positions, ctx.tok_entry, table, inv2, k2, v2, H, G, Dq, 16))
        note(f"rope_cache_{label}", ms, n * (H + 2 * G) * Dq * 2 * 2)

    # ---- feed-forward: group-routed experts with the clamped activation beside a dense SwiGLU of the width one token uses ----
    gu, dn = rnd(E, 2 * ff, d, k=0.05), rnd(E, d, ff, k=0.05)
    router, corr = rnd(E, d, k=0.1), rnd(E, dtype=torch.float32, k=0.1)
    dense_ff = top * ff
    wgu, wdn = rnd(2 * dense_ff, d, k=0.05), rnd(d, dense_ff, k=0.05)
    wup, wdown = rnd(z["dense"], d, k=0.05), rnd(d, z["dense"], k=0.05)
    act3 = ("glu_clamped", 7.0, 1.702)
    for label, n in (("prefill", T), ("decode", batch)):
        h = rnd(n, d)
        y = torch.empty(n, d, device=dev)
        route = Linear(router)
        idx, w = L.moe_select_grouped(route.forward(h, out_dtype=torch.float32), corr, E, top, *z["groups"])
        ms = timer(lambda: L.moe_select_grouped(route.forward(h, out_dtype=torch.float32), corr, E, top, *z["groups"]))
        note(f"moe_route_grouped_{label}", ms, 2.0 * (n * d + E * d))
        used = min(E, n * top)
        ms = timer(lambda: M.experts(h, gu, dn, idx, w, None, None, y, act3))
        note(f"moe_experts_clamped_{label}", ms, 2.0 * used * 3 * ff * d + 2.0 * n * d + 4.0 * n * d, 6.0 * n * top * ff * d)
        act = torch.empty(n, dense_ff, dtype=bf, device=dev)
        o = torch.empty(n, d, dtype=torch.float32, device=dev)

        def dense():
            if not tc_gemm.gemm_swiglu(h, wgu, act):
                K.swiglu(K.Partials(tc_gemm.partials(h, wgu)), act)
            tc_gemm.gemm(act, wdn, None, o)
        ms = timer(dense)
        note(f"dense_swiglu_{label}", ms, 2.0 * 3 * dense_ff * d + 6.0 * n * d, 6.0 * n * dense_ff * d)
        up, down = Linear(wup), Linear(wdown)
        a2 = torch.empty(n, z["dense"], dtype=bf, device=dev)

        def relu2():
            L.relu2(up.forward(h, defer=True), a2)
            r = down.forward(a2, defer=True, residual=True)
            if isinstance(r, K.Partials):
                r.materialize(torch.float32)
        ms = timer(relu2)
        note(f"dense_relu2_{label}", ms, 2.0 * 2 * z["dense"] * d + 6.0 * n * d, 4.0 * n * z["dense"] * d)

    # ---- the residual: one pass over S streams beside add + RMSNorm over one -------------------------------------------
    for label, n in (("prefill", T), ("decode", batch)):
        xs, yv = rnd(n, S, d, dtype=torch.float32), rnd(n, d, dtype=torch.float32)
        mix, wo, wi = rnd(S, S, dtype=torch.float32), rnd(S, dtype=torch.float32), rnd(S, dtype=torch.float32)
        nw, hb = torch.ones(d, device=dev), torch.empty(n, d, dtype=bf, device=dev)
        ms = timer(lambda: L.hyper_step(xs, yv, mix, wo, wi, nw, 1e-5, hb))
        note(f"hyper_step_{label}", ms, n * d * (8.0 * S + 4 + 2))
        x = rnd(n, d, dtype=torch.float32)
        ms = timer(lambda: K.add_rmsnorm(x, yv, nw, 1e-5, hb))
        note(f"add_rmsnorm_{label}", ms, n * d * (4 + 4 + 4 + 2))
    return rows


def time_banelix_kernels(z, T, context, batch, timer, peaks):
    """Banelix's kernels alone, each beside the kernel of the built-in decoder that does the like job."""
    import numpy as np
    import torch
    from infero_b200 import kernels as K
    from infero_b200.kernels import attention as A, layer_ops as L
    dev, bf = "cuda:0", torch.bfloat16
    d, H, G, D, W, C, nb, taps = z["width"], z["heads"], z["kv"], z["dim"], z["window"], z["rec"], z["blocks"], z["taps"]
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf, k=1.0: (torch.randn(s, generator=g, device=dev) * k).to(dtype)     # noqa: E731
    i32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.int32, device=dev)                 # noqa: E731
    hbm, tfl = peaks["hbm_gbs"], peaks["bf16_tflops"]
    rows = {}

    def note(name, ms, bytes_=0.0, flops=0.0, **more):
        r = {"us": round(ms * 1e3, 1)}
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["hbm_frac"] = round(bytes_ / ms / 1e6 / hbm, 3)
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 1)
            r["tensor_frac"] = round(flops / ms / 1e9 / tfl, 3)
        r.update(more)
        rows[name] = r

    def batch_ctx(q_lens, pos0, ps=16):
        E_ = len(q_lens)
        per = [-(-(p + n) // ps) for p, n in zip(pos0, q_lens)]
        table = torch.full((E_, max(per)), -1, dtype=torch.int32)
        at = 0
        for e, n in enumerate(per):
            table[e, :n] = torch.arange(at, at + n, dtype=torch.int32)
            at += n
        qs = np.concatenate([[0], np.cumsum(q_lens)[:-1]])
        ctx = types.SimpleNamespace(
            n_entries=E_, n_tokens=int(sum(q_lens)), h_q_len=np.asarray(q_lens, dtype=np.int32), h_pos0=np.asarray(pos0, dtype=np.int32),
            tok_entry=i32(np.repeat(np.arange(E_), q_lens)), positions=i32(np.concatenate([p + np.arange(n) for p, n in zip(pos0, q_lens)])),
            entry_q_start=i32(qs), entry_q_len=i32(q_lens), entry_pos0=i32(pos0), entry_slot=i32(np.arange(E_)), kv_bound=None)
        return ctx, table.to(dev), at

    for label, q_lens, pos0 in (("prefill", [T], [0]), ("decode", [1] * batch, [context - 1] * batch)):
        ctx, table, pages = batch_ctx(q_lens, pos0)
        n = ctx.n_tokens
        # ---- attention: a window and a sink beside all keys and none -----------------------------------------------
        kc, vc = rnd(pages, G, 16, D), rnd(pages, G, 16, D)
        q, out = rnd(n, H * D), torch.empty(n, H * D, dtype=bf, device=dev)
        w = min(W, T if label == "prefill" else context)
        pairs_all = T * T / 2 if label == "prefill" else batch * context
        pairs_win = (T * w - w * w / 2) if label == "prefill" else batch * w
        keys_all = T if label == "prefill" else batch * context
        keys_win = T if label == "prefill" else batch * w
        for name, window, sink, pairs, keys in (("window_sink_attention", W, True, pairs_win, keys_win),
                                                ("gqa_attention", None, False, pairs_all, keys_all)):
            ms = timer(lambda: A.attention_any(q, out, kc, vc, table, ctx.tok_entry, ctx.positions, H, G, D, 16, window, D ** -0.5,
                                               ctx.h_q_len, ctx.h_pos0, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_pos0, sink=sink))
            note(f"{name}_{label}", ms, 2.0 * G * 2 * D * keys + 4.0 * n * H * D, 2.0 * H * 2 * D * pairs)
        # ---- from the input product to queries and the cache: both norms beside rotary + cache append ---------------------
        width = (H + 2 * G) * D
        proj = rnd(n, width, dtype=torch.float32)
        qo = torch.empty(n, H * D, dtype=bf, device=dev)
        fr = torch.rand(D // 2, device=dev, dtype=torch.float64)
        qw, kw = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
        ms = timer(lambda: L.qk_prepare(proj, 0, H * D, (H + G) * D, 1, qw, kw, 1e-5, fr, 1.1, ctx.positions, ctx.tok_entry, table,
                                        16, qo, kc, vc, H, G, D, D))
        note(f"qk_prepare_projection_norm_{label}", ms, n * width * (4.0 + 2.0))
        ms = timer(lambda: L.qk_prepare(proj, 0, H * D, -1, 2, None, None, 1e-5, fr, 1.0, ctx.positions, ctx.tok_entry, table,
                                        16, qo, kc, vc, H, G, D, D))
        note(f"qk_prepare_head_norm_{label}", ms, n * (H + G) * D * 4.0 + n * (H + 2 * G) * D * 2.0)
        qkv = rnd(n, width)
        inv = torch.rand(D // 2, device=dev)
        ms = timer(lambda: K.rope_cache(qkv, ctx.positions, ctx.tok_entry, table, inv, kc, vc, H, G, D, 16))
        note(f"rope_cache_{label}", ms, n * width * 2 * 2)
        # ---- the gate per head ---------------------------------------------------------------------------------------
        gate = rnd(n, H, dtype=torch.float32)
        ms = timer(lambda: L.head_gate(out, gate, out, H, D, 0.7))
        note(f"head_gate_{label}", ms, n * H * D * 4.0 + n * H * 4.0)
        # ---- the recurrence: convolution, gate products and scan ------------------------------------------------------
        rctx, _, _ = batch_ctx(q_lens, [0] * len(q_lens))
        bs = C // nb
        yx = rnd(n, 2 * C, dtype=torch.float32)
        cw, cb = rnd(C, taps, dtype=torch.float32, k=0.3), rnd(C, dtype=torch.float32, k=0.1)
        cwt = cw.t().contiguous()
        wg = rnd(nb, 2 * bs, bs, k=bs ** -0.5)
        rb, ib, lam = rnd(C, dtype=torch.float32, k=0.1), rnd(C, dtype=torch.float32, k=0.1), rnd(C, dtype=torch.float32)
        state = torch.zeros(len(q_lens), taps, C, device=dev)
        ro = torch.empty(n, C, dtype=bf, device=dev)
        ms = timer(lambda: L.rglru(yx, 0, C, cw, cb, wg, rb, ib, lam, 8.0, state, rctx.tok_entry, rctx.entry_q_start, rctx.entry_q_len,
                                   rctx.entry_slot, len(q_lens), ro, 0.7, max_q_len=max(q_lens), tensor_cores=True, conv_wt=cwt))
        least = n * C * (8.0 + 2.0) + 2.0 * wg.numel() + 8.0 * len(q_lens) * taps * C
        moved = least + n * C * (4.0 + 2.0 + 4.0 + 8.0 + 8.0 + 4.0)           # u written and read twice (+ bf16), gates written and read
        note(f"rglru_{label}", ms, least, 2.0 * n * 2 * C * bs, gb_s_with_intermediates=round(moved / ms / 1e6, 1),
             hbm_frac_with_intermediates=round(moved / ms / 1e6 / hbm, 3))
        # ---- add + RMSNorm with the sublayer's result times a constant (the same kernel as without) -----------------------
        x, yv = rnd(n, d, dtype=torch.float32), rnd(n, d, dtype=torch.float32)
        nw, hb = torch.ones(d, device=dev), torch.empty(n, d, dtype=bf, device=dev)
        ms = timer(lambda: K.add_rmsnorm(x, yv, nw, 1e-5, hb, delta_scale=0.5))
        note(f"add_rmsnorm_scaled_{label}", ms, n * d * (4 + 4 + 4 + 2))
    return rows


def time_pibavik_kernels(z, T, context, batch, timer, peaks):
    """Pibavik's kernels alone, each beside the kernel of another design that does the like job."""
    import numpy as np
    import torch
    from infero_b200 import kernels as K
    from infero_b200.kernels import attention as A, layer_ops as L, moe as M
    dev, bf = "cuda:0", torch.bfloat16
    d, H, G, D, W = z["width"], z["heads"], z["kv"], z["dim"], z["window"]
    Hn, P, N, Gs, taps, parts = z["ssd_heads"], z["ssd_vdim"], z["state"], z["groups"], z["taps"], z["norm_groups"]
    E, top, ff = z["experts"], z["top"], z["ff"]
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf, k=1.0: (torch.randn(s, generator=g, device=dev) * k).to(dtype)     # noqa: E731
    i32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.int32, device=dev)                 # noqa: E731
    hbm, tfl = peaks["hbm_gbs"], peaks["bf16_tflops"]
    rows = {}

    def note(name, ms, bytes_=0.0, flops=0.0, **more):
        r = {"us": round(ms * 1e3, 1)}
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["hbm_frac"] = round(bytes_ / ms / 1e6 / hbm, 3)
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 1)
            r["tensor_frac"] = round(flops / ms / 1e9 / tfl, 3)
        r.update(more)
        rows[name] = r

    def batch_ctx(q_lens, pos0, ps=16):
        E_ = len(q_lens)
        per = [-(-(p + n) // ps) for p, n in zip(pos0, q_lens)]
        table = torch.full((E_, max(per)), -1, dtype=torch.int32)
        at = 0
        for e, n in enumerate(per):
            table[e, :n] = torch.arange(at, at + n, dtype=torch.int32)
            at += n
        qs = np.concatenate([[0], np.cumsum(q_lens)[:-1]])
        ctx = types.SimpleNamespace(
            n_entries=E_, n_tokens=int(sum(q_lens)), h_q_len=np.asarray(q_lens, dtype=np.int32), h_pos0=np.asarray(pos0, dtype=np.int32),
            tok_entry=i32(np.repeat(np.arange(E_), q_lens)), positions=i32(np.concatenate([p + np.arange(n) for p, n in zip(pos0, q_lens)])),
            entry_q_start=i32(qs), entry_q_len=i32(q_lens), entry_pos0=i32(pos0), entry_slot=i32(np.arange(E_)), kv_bound=None)
        return ctx, table.to(dev), at

    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=torch.float32, device=dev)
    for label, q_lens, pos0 in (("prefill", [T], [0]), ("decode", [1] * batch, [context - 1] * batch)):
        ctx, table, pages = batch_ctx(q_lens, pos0)
        n = ctx.n_tokens
        # ---- window attention with a distance bias beside window attention with a sink -------------------------------
        kc, vc = rnd(pages, G, 16, D), rnd(pages, G, 16, D)
        q, out = rnd(n, H * D), torch.empty(n, H * D, dtype=bf, device=dev)
        w = min(W, T if label == "prefill" else context)
        pairs = (T * w - w * w / 2) if label == "prefill" else batch * w
        keys = T if label == "prefill" else batch * w
        for name, sink, sl in (("window_bias_attention", False, slopes), ("window_sink_attention", True, None)):
            ms = timer(lambda: A.attention_any(q, out, kc, vc, table, ctx.tok_entry, ctx.positions, H, G, D, 16, W, D ** -0.5,
                                               ctx.h_q_len, ctx.h_pos0, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_pos0,
                                               sink=sink, slopes=sl))
            note(f"{name}_{label}", ms, 2.0 * G * 2 * D * keys + 4.0 * n * H * D, 2.0 * H * 2 * D * pairs)
        # ---- from the input product to queries and the cache: the norm per head beside the norm over the projection ------
        width = (H + 2 * G) * D
        proj = rnd(n, width, dtype=torch.float32)
        qo = torch.empty(n, H * D, dtype=bf, device=dev)
        fr = torch.rand(D // 4, device=dev, dtype=torch.float64)
        for name, mode, qw, kw in (("qk_prepare_weighted_head_norm", 3, torch.ones(D, device=dev), torch.ones(D, device=dev)),
                                   ("qk_prepare_projection_norm", 1, torch.ones(H * D, device=dev), torch.ones(G * D, device=dev))):
            ms = timer(lambda: L.qk_prepare(proj, 0, H * D, (H + G) * D, mode, qw, kw, 1e-5, fr, 1.0, ctx.positions, ctx.tok_entry,
                                            table, 16, qo, kc, vc, H, G, D, D))
            note(f"{name}_{label}", ms, n * width * (4.0 + 2.0))
        # ---- the state-space recurrence beside the gated linear recurrence of equal width -----------------------------
        rctx, _, _ = batch_ctx(q_lens, [0] * len(q_lens))
        inner, CH = Hn * P, Hn * P + 2 * Gs * N
        zx = rnd(n, 2 * inner + 2 * Gs * N + Hn, dtype=torch.float32, k=0.5)
        cw, cb = rnd(CH, taps, dtype=torch.float32, k=0.3), rnd(CH, dtype=torch.float32, k=0.1)
        dtb, alog, skip = rnd(Hn, dtype=torch.float32) - 3.0, rnd(Hn, dtype=torch.float32, k=0.2), rnd(Hn, dtype=torch.float32)
        nw = torch.ones(inner, device=dev)
        state = torch.zeros(len(q_lens), L.ssd_state_floats(Hn, N, P, Gs, taps), device=dev)
        so = torch.empty(n, inner, dtype=bf, device=dev)
        ms = timer(lambda: L.ssd(zx, 0, inner, inner + CH, cw, cb, dtb, alog, skip, nw, 1e-5, parts, state, rctx.tok_entry,
                                 rctx.entry_q_start, rctx.entry_q_len, rctx.entry_slot, len(q_lens), so, Hn, Gs, N, P, 0.7,
                                 max_q_len=max(q_lens)))
        least = n * (zx.shape[1] * 4.0 + inner * 2.0) + 8.0 * state.numel()
        moved = least + n * (CH * 8.0 + inner * 8.0)                       # the convolution's result and y written and read
        note(f"ssd_{label}", ms, least, 2.0 * n * Hn * N * P * 2, gb_s_with_intermediates=round(moved / ms / 1e6, 1),
             hbm_frac_with_intermediates=round(moved / ms / 1e6 / hbm, 3))
        C, nb = inner, H
        bs = C // nb
        yx = rnd(n, 2 * C, dtype=torch.float32)
        rw, rb_ = rnd(C, taps, dtype=torch.float32, k=0.3), rnd(C, dtype=torch.float32, k=0.1)
        wg = rnd(nb, 2 * bs, bs, k=bs ** -0.5)
        rb, ib, lam = rnd(C, dtype=torch.float32, k=0.1), rnd(C, dtype=torch.float32, k=0.1), rnd(C, dtype=torch.float32)
        rstate = torch.zeros(len(q_lens), taps, C, device=dev)
        ro = torch.empty(n, C, dtype=bf, device=dev)
        ms = timer(lambda: L.rglru(yx, 0, C, rw, rb_, wg, rb, ib, lam, 8.0, rstate, rctx.tok_entry, rctx.entry_q_start, rctx.entry_q_len,
                                   rctx.entry_slot, len(q_lens), ro, 0.7, max_q_len=max(q_lens), tensor_cores=True))
        note(f"rglru_{label}", ms, n * C * (8.0 + 2.0) + 2.0 * wg.numel() + 8.0 * len(q_lens) * taps * C, 2.0 * n * 2 * C * bs)
        # ---- ungated experts that read their weighted input beside gated experts of the same sizes --------------------
        h = rnd(n, d)
        up, down = rnd(E, ff, d, k=d ** -0.5), rnd(E, d, ff, k=ff ** -0.5)
        gate_up = rnd(E, 2 * ff, d, k=d ** -0.5)
        logits = rnd(n, E, dtype=torch.float32)
        idx, wts = L.moe_select_scored(logits, E, top)
        y = torch.empty(n, d, dtype=torch.float32, device=dev)
        touched = min(E, n * top)
        ms = timer(lambda: M.plain_experts(h, up, down, idx, wts, True, None, y))
        note(f"experts_relu2_weighted_input_{label}", ms, touched * 2.0 * ff * d * 2 + n * d * (2.0 + 4.0), 2.0 * n * top * 2 * ff * d)
        ms = timer(lambda: M.experts(h, gate_up, down, idx, wts, None, None, y))
        note(f"experts_swiglu_{label}", ms, touched * 3.0 * ff * d * 2 + n * d * (2.0 + 4.0), 2.0 * n * top * 3 * ff * d)
        ms = timer(lambda: L.moe_select_scored(logits, E, top))
        note(f"select_by_sigmoid_scores_{label}", ms, n * E * 4.0 + n * top * 8.0)
        ms = timer(lambda: L.moe_select(logits, E, top))
        note(f"select_by_softmax_of_chosen_{label}", ms, n * E * 4.0 + n * top * 8.0)
        # ---- the norm of a column slice (the queries' latent) beside add + RMSNorm ------------------------------------
        Q = z["q_rank"]
        wide = rnd(n, Q + z["kv_rank"], dtype=torch.float32)
        cq = torch.empty(n, Q, dtype=bf, device=dev)
        qn = torch.ones(Q, device=dev)
        ms = timer(lambda: L.gated_group_norm(wide[:, :Q], None, qn, 1e-5, 1, cq))
        note(f"latent_query_norm_{label}", ms, n * Q * (4.0 + 2.0))
        x, yv = rnd(n, d, dtype=torch.float32), rnd(n, d, dtype=torch.float32)
        nw2, hb = torch.ones(d, device=dev), torch.empty(n, d, dtype=bf, device=dev)
        ms = timer(lambda: K.add_rmsnorm(x, yv, nw2, 1e-5, hb))
        note(f"add_rmsnorm_{label}", ms, n * d * (4 + 4 + 4 + 2))
    return rows


def time_nuvarax_kernels(z, T, context, batch, timer, peaks):
    """Nuvarax's kernels alone, each beside the kernel of another design that does the like job."""
    import numpy as np
    import torch
    from infero_b200 import kernels as K
    from infero_b200.kernels import attention as A, layer_ops as L
    from infero_b200.parts.normed_attention import distance_buckets
    dev, bf, f32 = "cuda:0", torch.bfloat16, torch.float32
    d, H, G, D = z["width"], z["heads"], z["kv"], z["dim"]
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf, k=1.0: (torch.randn(s, generator=g, device=dev) * k).to(dtype)     # noqa: E731
    i32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.int32, device=dev)                 # noqa: E731
    hbm, tfl = peaks["hbm_gbs"], peaks["bf16_tflops"]
    rows = {}

    def note(name, ms, bytes_=0.0, flops=0.0, **more):
        r = {"us": round(ms * 1e3, 1)}
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["hbm_frac"] = round(bytes_ / ms / 1e6 / hbm, 3)
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 1)
            r["tensor_frac"] = round(flops / ms / 1e9 / tfl, 3)
        r.update(more)
        rows[name] = r
        print(f"[design_bench] {name}: {json.dumps(r)}", file=sys.stderr, flush=True)

    def batch_ctx(q_lens, pos0, ps=16):
        E_ = len(q_lens)
        per = [-(-(p + n) // ps) for p, n in zip(pos0, q_lens)]
        table = torch.full((E_, max(per)), -1, dtype=torch.int32)
        at = 0
        for e, n in enumerate(per):
            table[e, :n] = torch.arange(at, at + n, dtype=torch.int32)
            at += n
        qs = np.concatenate([[0], np.cumsum(q_lens)[:-1]])
        ctx = types.SimpleNamespace(
            n_entries=E_, n_tokens=int(sum(q_lens)), max_q_len=max(q_lens), h_q_len=np.asarray(q_lens, dtype=np.int32),
            h_pos0=np.asarray(pos0, dtype=np.int32), tok_entry=i32(np.repeat(np.arange(E_), q_lens)),
            positions=i32(np.concatenate([p + np.arange(n) for p, n in zip(pos0, q_lens)])), entry_q_start=i32(qs),
            entry_q_len=i32(q_lens), entry_pos0=i32(pos0), entry_slot=i32(np.arange(E_)), kv_bound=None)
        return ctx, table.to(dev), at

    buckets = distance_buckets(32, z["bias_max"])
    rel = rnd(H, len(buckets), dtype=f32)
    rel2 = rel * 1.4426950408889634
    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=f32, device=dev)
    for label, q_lens, pos0 in (("prefill", [T], [0]), ("decode", [1] * batch, [context - 1] * batch)):
        ctx, table, pages = batch_ctx(q_lens, pos0)
        n, single = ctx.n_tokens, label == "decode"
        # ---- attention with a learned distance bias and mixed heads beside attention with a distance slope -----------
        kc, vc = rnd(pages, G, 16, D), rnd(pages, G, 16, D)
        kv = types.SimpleNamespace(k=kc, v=vc, page_size=16, group=0)
        q, out = rnd(n, H * D), torch.empty(n, H * D, dtype=bf, device=dev)
        pairs = T * (T + 1) / 2 if label == "prefill" else batch * context
        keys = T if label == "prefill" else batch * context
        bytes_ = 2.0 * G * 2 * D * keys + 4.0 * n * H * D
        flops = 2.0 * H * 2 * D * pairs
        mix, gate = rnd(H, H, dtype=f32), rnd(n, H * D, dtype=f32)

        def mixed():
            a = A.paged_attention_cross(ctx, q, kv, table, H, G, D, D, None, D ** -0.5, rel=rel, rel_log2=rel2)
            L.head_mix(a, mix, gate, out, H, G, D)
        note(f"mixed_head_attention_{label}", timer(mixed), bytes_, flops)
        a = A.paged_attention_cross(ctx, q, kv, table, H, G, D, D, None, D ** -0.5, rel=rel, rel_log2=rel2)
        note(f"head_mix_{label}", timer(lambda: L.head_mix(a, mix, gate, out, H, G, D)),
             n * (a.shape[1] * a.element_size() + H * D * 6.0))
        ms = timer(lambda: A.attention_any(q, out, kc, vc, table, ctx.tok_entry, ctx.positions, H, G, D, 16, None, D ** -0.5, ctx.h_q_len,
                                           ctx.h_pos0, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_pos0, slopes=slopes))
        note(f"slope_bias_attention_{label}", ms, bytes_, flops)
        # ---- the two memories beside the state-space recurrence of as many state numbers ------------------------------
        rctx, _, _ = batch_ctx(q_lens, [0] * len(q_lens))
        E = len(q_lens)
        Hd, Gd, Kd, Vd, taps = z["delta_heads"], z["delta_kv"], z["delta_dim"], z["delta_vdim"], z["taps"]
        CH = 2 * Gd * Kd + Hd * Vd
        proj = rnd(n, CH + Hd * Vd + 2 * Hd, dtype=f32, k=0.5)
        cw, alog, dtb, nw = rnd(taps, CH, dtype=f32, k=0.4), rnd(Hd, dtype=f32, k=0.2), rnd(Hd, dtype=f32) - 3.0, torch.ones(Vd, device=dev)
        state = torch.zeros(E, L.memory_state_floats("delta", Hd, Kd, Vd, taps, CH), device=dev)
        so, dout = L.memory_tail_floats(taps, CH), torch.empty(n, Hd * Vd, dtype=bf, device=dev)
        args = (rctx.entry_q_start, rctx.entry_q_len, rctx.entry_slot, E)

        def prepare():
            return L.memory_prepare(proj, 0, CH + Hd * Vd + Hd, CH + Hd * Vd, cw, alog, dtb, state, rctx.tok_entry, *args, Gd, Hd, Kd, Vd, single)
        u, table_ = prepare()

        def scan():
            return L.delta_scan(u, table_, state, so, *args, Hd, Gd, Kd, Vd, single)
        y = scan()

        def finish():
            L.memory_finish(y, None, proj[:, CH:CH + Hd * Vd], "silu", nw, 1e-5, dout, Hd, Vd)
        least = n * (proj.shape[1] * 4.0 + Hd * Vd * 2.0) + 8.0 * state.numel()
        note(f"delta_memory_{label}", timer(lambda: (prepare(), scan(), finish())), least, 2.0 * n * Hd * Kd * Vd * 3)
        note(f"memory_prepare_{label}", timer(prepare), n * CH * 8.0)
        note(f"memory_scan_delta_{label}", timer(scan), n * (CH + Hd * Vd) * 4.0 + 8.0 * E * Hd * Kd * Vd, 2.0 * n * Hd * Kd * Vd * 3)
        note(f"memory_finish_{label}", timer(finish), n * Hd * Vd * 10.0)
        Hm, Km, Vm = z["mem_heads"], z["mem_dim"], z["mem_vdim"]
        gw = 2 * Hm * Km + 2 * Hm * Vm + 2 * Hm
        gp, gn = rnd(n, gw, dtype=f32, k=0.5), torch.ones(Hm * Vm, device=dev)
        gstate, gout = torch.zeros(E, L.memory_state_floats("gated", Hm, Km, Vm), device=dev), torch.empty(n, Hm * Vm, dtype=bf, device=dev)
        v0 = 2 * Hm * Km

        def gated():
            y_, den = L.gated_scan(gp, 0, Hm * Km, v0, v0 + 2 * Hm * Vm, v0 + 2 * Hm * Vm + Hm, 15.0, gstate, 0, *args, Hm, Km, Vm, single)
            L.memory_finish(y_, den, gp[:, v0 + Hm * Vm:v0 + 2 * Hm * Vm], "sigmoid", gn, 1e-5, gout, Hm, Vm)
        note(f"gated_memory_{label}", timer(gated), n * (gw * 4.0 + Hm * Vm * 2.0) + 8.0 * gstate.numel(), 2.0 * n * Hm * Km * Vm * 2)
        P, N = 64, Km
        Hn, Gs = Hm * Vm // P, max(1, Hm * Vm // P // 8)
        inner, C2 = Hn * P, Hn * P + 2 * Gs * N
        zx = rnd(n, 2 * inner + 2 * Gs * N + Hn, dtype=f32, k=0.5)
        cw2, cb2 = rnd(C2, taps, dtype=f32, k=0.3), rnd(C2, dtype=f32, k=0.1)
        sstate, so2 = torch.zeros(E, L.ssd_state_floats(Hn, N, P, Gs, taps), device=dev), torch.empty(n, inner, dtype=bf, device=dev)
        sdt, sal, skip, snw = rnd(Hn, dtype=f32), rnd(Hn, dtype=f32, k=0.2), rnd(Hn, dtype=f32), torch.ones(inner, device=dev)
        ms = timer(lambda: L.ssd(zx, 0, inner, inner + C2, cw2, cb2, sdt, sal, skip, snw, 1e-5, Gs, sstate, rctx.tok_entry, rctx.entry_q_start, rctx.entry_q_len,
                                 rctx.entry_slot, E, so2, Hn, Gs, N, P, 0.7, max_q_len=max(q_lens)))
        note(f"ssd_{label}", ms, n * (zx.shape[1] * 4.0 + inner * 2.0) + 8.0 * sstate.numel(), 2.0 * n * Hn * N * P * 2)
        # ---- norms around a sublayer beside add + RMSNorm; the input convolution -------------------------------------
        x, yv, y2 = rnd(n, d, dtype=f32), rnd(n, d, dtype=f32), rnd(n, d, dtype=f32)
        w1, hb, hf = torch.ones(d, device=dev), torch.empty(n, d, dtype=bf, device=dev), torch.empty(n, d, dtype=f32, device=dev)
        one, two = K.NormedDelta(yv, w1, 1e-5), K.NormedDelta(K.BranchSum([yv, y2], [w1, w1], 1e-5, 0.5), w1, 1e-5)
        note(f"sandwich_norm_{label}", timer(lambda: L.sandwich_norm(x, one, w1, 1e-5, hb)), n * d * (4 + 4 + 4 + 2.0))
        note(f"sandwich_norm_two_branches_{label}", timer(lambda: L.sandwich_norm(x, two, w1, 1e-5, hb)), n * d * (4 + 4 + 4 + 4 + 2.0))
        note(f"add_rmsnorm_{label}", timer(lambda: K.add_rmsnorm(x, yv, w1, 1e-5, hb)), n * d * (4 + 4 + 4 + 2.0))
        cw4, cstate = rnd(4, d, dtype=f32, k=0.3), torch.zeros(E, 3 * d, device=dev)
        if single:
            note("sandwich_norm_with_conv_decode", timer(lambda: L.sandwich_norm(x, one, w1, 1e-5, hb, conv=(cw4, cstate, rctx.tok_entry, rctx.entry_slot))),
                 n * d * (4 + 4 + 4 + 2.0 + 24))
        else:
            note("input_conv_prefill", timer(lambda: L.input_conv(hf, cw4, cstate, rctx.tok_entry, *args, hb)), n * d * 6.0)
        tab, big, pos = rnd(z["vocab"], d), rnd(2 * z["vocab"] + 2, d), rnd(4096, d)
        ids, prev = i32(np.arange(n) % z["vocab"]), torch.zeros(E, 1, dtype=torch.int32, device=dev)
        note(f"embed_compose_{label}", timer(lambda: L.embed_compose(tab, ids, x, 1.0, None, (big, 2 * z["vocab"] + 1, 31, 17), prev, pos,
                                                                    rctx.positions, rctx.tok_entry, *args, single)), n * d * 10.0)
        note(f"embed_gather_{label}", timer(lambda: K.embed_gather(tab, ids, x)), n * d * 6.0)
    return rows


def time_dukolorn_kernels(z, T, context, batch, timer, peaks):
    """Dukolorn's kernels alone, each beside the kernel of another design that does the like job."""
    import numpy as np
    import torch
    from infero_b200 import kernels as K
    from infero_b200.kernels import attention as A, latent_attention as LA, layer_ops as L
    from infero_b200.parts.linear import Linear
    from infero_b200.parts.normed_attention import distance_buckets
    dev, bf, f32 = "cuda:0", torch.bfloat16, torch.float32
    d, H, G, D = z["width"], z["heads"], z["kv"], z["dim"]
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf, k=1.0: (torch.randn(s, generator=g, device=dev) * k).to(dtype)     # noqa: E731
    i32 = lambda a: torch.tensor(np.asarray(a), dtype=torch.int32, device=dev)                 # noqa: E731
    hbm, tfl = peaks["hbm_gbs"], peaks["bf16_tflops"]
    rows = {}

    def note(name, ms, bytes_=0.0, flops=0.0):
        r = {"us": round(ms * 1e3, 1)}
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["hbm_frac"] = round(bytes_ / ms / 1e6 / hbm, 3)
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 1)
            r["tensor_frac"] = round(flops / ms / 1e9 / tfl, 3)
        rows[name] = r
        print(f"[design_bench] {name}: {json.dumps(r)}", file=sys.stderr, flush=True)

    def batch_ctx(q_lens, pos0, ps=16):
        E_ = len(q_lens)
        per = [-(-(p + n) // ps) for p, n in zip(pos0, q_lens)]
        table = torch.full((E_, max(per)), -1, dtype=torch.int32)
        at = 0
        for e, n in enumerate(per):
            table[e, :n] = torch.arange(at, at + n, dtype=torch.int32)
            at += n
        qs = np.concatenate([[0], np.cumsum(q_lens)[:-1]])
        ctx = types.SimpleNamespace(
            n_entries=E_, n_tokens=int(sum(q_lens)), max_q_len=max(q_lens), h_q_len=np.asarray(q_lens, dtype=np.int32),
            h_pos0=np.asarray(pos0, dtype=np.int32), tok_entry=i32(np.repeat(np.arange(E_), q_lens)),
            positions=i32(np.concatenate([p + np.arange(n) for p, n in zip(pos0, q_lens)])), entry_q_start=i32(qs),
            entry_q_len=i32(q_lens), entry_pos0=i32(pos0), entry_slot=i32(np.arange(E_)), kv_bound=None)
        return ctx, table.to(dev), at

    rel = rnd(H, len(distance_buckets(32, z["bias_max"])), dtype=f32)
    sinks, slopes = rnd(H, dtype=f32), torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=f32, device=dev)
    rel2, sinks2 = rel * A.LOG2E, sinks * A.LOG2E
    for label, q_lens, pos0 in (("prefill", [T], [0]), ("decode", [1] * batch, [context - 1] * batch)):
        ctx, table, pages = batch_ctx(q_lens, pos0)
        n, single = ctx.n_tokens, label == "decode"
        # ---- attention with a soft cap, a distance table and sinks beside attention with a distance slope ----------
        kc, vc = rnd(pages, G, 16, D), rnd(pages, G, 16, D)
        kv = types.SimpleNamespace(k=kc, v=vc, page_size=16, group=0)
        q, out = rnd(n, H * D), torch.empty(n, H * D, dtype=bf, device=dev)
        pairs = T * (T + 1) / 2 if not single else batch * context
        keys = T if not single else batch * context
        bytes_, flops = 2.0 * G * 2 * D * keys + 4.0 * n * H * D, 2.0 * H * 2 * D * pairs
        attend = lambda **kw: A.paged_attention_ex(ctx, q, out, kv, table, H, G, D, D, None, D ** -0.5, False, **kw)       # noqa: E731
        note(f"capped_attention_{label}", timer(lambda: attend(rel=rel, rel_log2=rel2, sinks=sinks, sinks_log2=sinks2, softcap=30.0)), bytes_, flops)
        note(f"table_bias_attention_{label}", timer(lambda: attend(rel=rel, rel_log2=rel2)), bytes_, flops)
        note(f"slope_bias_attention_{label}", timer(lambda: attend(slopes=slopes)), bytes_, flops)
        proj, qw, kw = rnd(n, (H + 2 * G) * D, dtype=f32), torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
        prep = lambda **kw2: L.qk_prepare(proj, 0, H * D, (H + G) * D, 1, qw, kw, 1e-5, None, 1.0, ctx.positions, ctx.tok_entry, table, 16, q,   # noqa: E731
                                          kc, vc, H, G, D, D, **kw2)
        note(f"qk_prepare_temperature_{label}", timer(lambda: prep(temperature=(0.1, 1024), v_scale=0.9)), n * (H + 2 * G) * D * 6.0)
        note(f"qk_prepare_{label}", timer(prep), n * (H + 2 * G) * D * 6.0)
        # ---- the memories with decays per channel beside those with one per head -----------------------------------
        rctx, _, _ = batch_ctx(q_lens, [0] * len(q_lens))
        E, rank = len(q_lens), 64
        args = (rctx.entry_q_start, rctx.entry_q_len, rctx.entry_slot, E)
        Hd, Gd, Kd, Vd, taps = z["delta_heads"], z["delta_kv"], z["delta_dim"], z["delta_vdim"], z["taps"]
        CH = 2 * Gd * Kd + Hd * Vd
        cw, alog, nw = rnd(taps, CH, dtype=f32, k=0.4), rnd(Hd, dtype=f32, k=0.2), torch.ones(Vd, device=dev)
        dtb, dtc = rnd(Hd, dtype=f32) - 3.0, rnd(Hd * Kd, dtype=f32) - 3.0
        cp = rnd(n, CH + 2 * rank + Hd, dtype=f32, k=0.5)
        a2, g2 = rnd(Hd * Kd, rank, k=0.1), rnd(Hd * Vd, rank, k=0.1)
        state = torch.zeros(E, L.memory_state_floats("delta", Hd, Kd, Vd, taps, CH), device=dev)
        so, dout = L.memory_tail_floats(taps, CH), torch.empty(n, Hd * Vd, dtype=bf, device=dev)
        narrow = lambda: L.low_rank(cp[:, CH:CH + rank], a2, "decay", dtc, alog, beside=(cp[:, CH + rank:CH + 2 * rank], g2))       # noqa: E731
        decay, gate = narrow()
        cprep = lambda dec: L.channel_prepare(cp, 0, CH + 2 * rank, cw, dec, state, rctx.tok_entry, *args, Gd, Hd, Kd, Vd, single)       # noqa: E731
        u, tab = cprep(decay)
        cscan = lambda u_, t_: L.channel_scan(u_, t_, state, so, *args, Hd, Kd, Vd, single)       # noqa: E731
        y = cscan(u, tab)

        def whole_channel():
            dec, gt = narrow()
            L.memory_finish(cscan(*cprep(dec)), None, gt, "sigmoid", nw, 1e-5, dout, Hd, Vd)
        least = n * (cp.shape[1] * 4.0 + Hd * Vd * 2.0) + 8.0 * state.numel()
        work = 2.0 * n * Hd * Kd * Vd * 3
        note(f"channel_delta_{label}", timer(whole_channel), least, work)
        note(f"low_rank_two_{label}", timer(narrow), n * (2.0 * rank + Hd * Kd + Hd * Vd) * 4.0)
        note(f"channel_prepare_{label}", timer(lambda: cprep(decay)), n * (CH + Hd * Kd + 3.25 * Hd * Kd + Hd * Vd) * 4.0)
        note(f"channel_scan_{label}", timer(lambda: cscan(u, tab)), n * (3.25 * Hd * Kd + 2 * Hd * Vd) * 4.0 + 8.0 * E * Hd * Kd * Vd, work)
        sp = rnd(n, CH + Hd * Vd + 2 * Hd, dtype=f32, k=0.5)
        sprep = lambda: L.memory_prepare(sp, 0, CH + Hd * Vd + Hd, CH + Hd * Vd, cw, alog, dtb, state, rctx.tok_entry, *args, Gd, Hd, Kd, Vd, single)   # noqa: E731
        su, st = sprep()
        sscan = lambda u_, t_: L.delta_scan(u_, t_, state, so, *args, Hd, Gd, Kd, Vd, single)       # noqa: E731

        def whole_delta():
            L.memory_finish(sscan(*sprep()), None, sp[:, CH:CH + Hd * Vd], "silu", nw, 1e-5, dout, Hd, Vd)
        note(f"delta_memory_{label}", timer(whole_delta), n * (sp.shape[1] * 4.0 + Hd * Vd * 2.0) + 8.0 * state.numel(), work)
        note(f"memory_prepare_{label}", timer(sprep), n * CH * 8.0)
        note(f"delta_scan_{label}", timer(lambda: sscan(su, st)), n * (CH + Hd * Vd) * 4.0 + 8.0 * E * Hd * Kd * Vd, work)
        Hm, Km, Vm = z["mem_heads"], z["mem_dim"], z["mem_vdim"]
        v0, gn = 2 * Hm * Km, torch.ones(Vm, device=dev)
        dp, w2, b2 = rnd(n, v0 + 2 * Hm * Vm + rank, dtype=f32, k=0.5), rnd(Hm * Km, rank, k=0.1), rnd(Hm * Km, dtype=f32) + 2.0
        mstate, mout = torch.zeros(E, L.memory_state_floats("gated", Hm, Km, Vm), device=dev), torch.empty(n, Hm * Vm, dtype=bf, device=dev)
        dstate = torch.zeros(E, L.memory_state_floats("delta", Hm, Km, Vm), device=dev)
        records = lambda: L.decayed_records(dp[:, v0 + 2 * Hm * Vm:], w2, b2, 16.0, dp, 0, Hm * Km, Hm, Km)       # noqa: E731
        dscan = lambda r: L.decayed_scan(dp[:, v0:v0 + Hm * Vm], r, dstate, 0, *args, Hm, Km, Vm, single)       # noqa: E731
        rec = records()

        def whole_decayed():
            L.memory_finish(dscan(records()), None, dp[:, v0 + Hm * Vm:v0 + 2 * Hm * Vm], "silu", gn, 1e-5, mout, Hm, Vm)
        mwork = 2.0 * n * Hm * Km * Vm * 2
        note(f"decayed_memory_{label}", timer(whole_decayed), n * (dp.shape[1] * 4.0 + Hm * Vm * 2.0) + 8.0 * dstate.numel(), mwork)
        note(f"decayed_records_{label}", timer(records), n * (5 * Hm * Km + rank) * 4.0)
        note(f"decayed_scan_{label}", timer(lambda: dscan(rec)), n * (3 * Hm * Km + 2 * Hm * Vm) * 4.0 + 8.0 * dstate.numel(), mwork)
        gp, gw = rnd(n, v0 + 2 * Hm * Vm + 2 * Hm, dtype=f32, k=0.5), torch.ones(Hm * Vm, device=dev)

        def whole_gated():
            y_, den = L.gated_scan(gp, 0, Hm * Km, v0, v0 + 2 * Hm * Vm, v0 + 2 * Hm * Vm + Hm, 15.0, mstate, 0, *args, Hm, Km, Vm, single)
            L.memory_finish(y_, den, gp[:, v0 + Hm * Vm:v0 + 2 * Hm * Vm], "sigmoid", gw, 1e-5, mout, Hm, Vm)
        note(f"gated_memory_{label}", timer(whole_gated), n * (gp.shape[1] * 4.0 + Hm * Vm * 2.0) + 8.0 * mstate.numel(), mwork)
        # ---- latent attention over a window with sinks beside latent attention over all keys -----------------------
        Hl, Dl, Rl, Vl, C, W = z["lat_heads"], z["lat_dim"], z["lat_rot"], z["lat_vdim"], z["lat_rank"], z["window"]
        lkv = types.SimpleNamespace(k=rnd(pages, 1, 16, C + Rl), v=None, page_size=16, group=0)
        rows_h = -(-n // 128) * 128
        q_lat, q_rot, o_lat = rnd(Hl, rows_h, C, dtype=f32), rnd(Hl, rows_h, Rl, dtype=f32), torch.empty(Hl, rows_h, C, dtype=bf, device=dev)
        lsink = rnd(Hl, dtype=f32)
        lsink2 = lsink * A.LOG2E
        seen = sum(min(i + 1, W) for i in range(T)) if not single else batch * min(context, W)
        for name, p, kk, kw2 in (("window_sink_latent", seen, T if not single else batch * min(context, W), dict(window=W, sinks=lsink, sinks_log2=lsink2)),
                                 ("latent", pairs, keys, {})):
            ms = timer(lambda: LA.attention(ctx, q_lat, q_rot, o_lat, lkv, table, n, Hl, C, Rl, (Dl + Rl) ** -0.5, **kw2))
            note(f"{name}_attention_{label}", ms, 2.0 * (C + Rl) * kk + n * Hl * (4.0 * (C + Rl) + 2.0 * C), 2.0 * Hl * (2 * C + Rl) * p)
        # ---- a norm on a sublayer's result beside norms on both sides; the embedding; the feed-forward ---------------
        x, yv, w1 = rnd(n, d, dtype=f32), rnd(n, d, dtype=f32), torch.ones(d, device=dev)
        hb = torch.empty(n, d, dtype=bf, device=dev)
        one = K.NormedDelta(yv, w1, 1e-5)
        note(f"post_norm_{label}", timer(lambda: L.sandwich_norm(x, one, None, 0.0, hb)), n * d * (4 + 4 + 4 + 2.0))
        note(f"sandwich_norm_{label}", timer(lambda: L.sandwich_norm(x, one, w1, 1e-5, hb)), n * d * (4 + 4 + 4 + 2.0))
        tabl, ids = rnd(z["vocab"], d), i32(np.arange(n) % z["vocab"])
        compose = lambda **kw2: L.embed_compose(tabl, ids, x, 1.0, None, None, None, None, rctx.positions, rctx.tok_entry, *args, single, **kw2)   # noqa: E731
        note(f"embed_norm_{label}", timer(lambda: compose(norm_w=w1, eps=1e-5, h=hb)), n * d * (2 + 4 + 2.0))
        note(f"embed_gather_{label}", timer(lambda: K.embed_gather(tabl, ids, x)), n * d * 6.0)
        ff = z["ff"]
        act, wgu, wdn, bgu = torch.empty(n, ff, dtype=bf, device=dev), rnd(2 * ff, d, k=0.02), rnd(d, ff, k=0.02), rnd(2 * ff, dtype=f32)
        for name, bias in (("biased_swiglu", bgu), ("swiglu", None)):
            lin, dn = Linear(wgu, bias), Linear(wdn, None)

            def mlp():
                if not lin.forward_swiglu(hb, act):
                    if bias is not None:
                        L.glu_act(lin.forward(hb, defer=True), act)
                    else:
                        K.swiglu(lin.forward(hb, defer=True), act)
                dn.forward(act, defer=True, residual=True)
            note(f"{name}_{label}", timer(mlp), 3.0 * d * ff * 2, 2.0 * n * 3 * d * ff)
    return rows


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="design_bench")
    ap.add_argument("--design", default="vufizen", choices=["vufizen", "gositar", "banelix", "pibavik", "nuvarax", "dukolorn"])
    ap.add_argument("--sizes", default="s,m")
    ap.add_argument("--prompt", type=int, default=2048)
    ap.add_argument("--context", type=int, default=2048)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=8)
    ap.add_argument("--kernels-at", default="m", help="the size whose kernels are timed alone ('' for none)")
    args = ap.parse_args(argv)
    import torch
    from infero_b200 import kernels as K
    K.lib()
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            m = json.load(f)
        peaks = {"hbm_gbs": float(m["hbm_gbs"]), "bf16_tflops": float(m["bf16_tflops"]), "source": "measured"}
    except (OSError, KeyError, ValueError):
        pass
    timer = _Timer()
    sizes, design_cfg, beside, each = {
        "vufizen": (SIZES, vufizen_config, {"qwen2": qwen2_config}, time_kernels),
        "gositar": (GOSITAR_SIZES, gositar_config, {"qwen2": qwen2_beside_gositar}, time_gositar_kernels),
        "banelix": (BANELIX_SIZES, banelix_config, {"qwen2": qwen2_beside_banelix}, time_banelix_kernels),
        "pibavik": (PIBAVIK_SIZES, pibavik_config, {"banelix": banelix_beside_pibavik}, time_pibavik_kernels),
        "nuvarax": (NUVARAX_SIZES, nuvarax_config, {"pibavik": lambda z, n: pibavik_config(PIBAVIK_SIZES[z["beside"]], n),
                                                    "banelix": lambda z, n: banelix_beside_pibavik(PIBAVIK_SIZES[z["beside"]], n)},
                    time_nuvarax_kernels),
        "dukolorn": (DUKOLORN_SIZES, dukolorn_config, {"nuvarax": nuvarax_config}, time_dukolorn_kernels)}[args.design]
    out = {"bench": "designs", "design": args.design, "dtype": "bf16", "data": "synthetic", "prompt": args.prompt, "context": args.context,
           "batch": args.batch, "layers": args.layers, "peaks": peaks, "sizes": {}}
    for name in [s for s in args.sizes.split(",") if s]:
        z = sizes[name]
        out["sizes"][name] = {"shape": z,
                              args.design: time_model(design_cfg(z, args.layers), args.prompt, args.context, args.batch, timer),
                              **{k: time_model(cfg(z, args.layers), args.prompt, args.context, args.batch, timer) for k, cfg in beside.items()}}
        print(f"[design_bench] {name}: {json.dumps(out['sizes'][name])}", file=sys.stderr, flush=True)
    if args.kernels_at:
        out["kernels"] = {"size": args.kernels_at,
                          "rows": each(sizes[args.kernels_at], args.prompt, args.context, args.batch, timer, peaks)}
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
