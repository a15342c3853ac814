"""Reading a Dukolorn config.json: what is accepted, what is refused, what the lowering makes of it (no GPU)."""
import copy

import pytest
import torch

import plain_dukolorn as PD
from dukolorn_fixtures import BUCKETS, CONFIGS, RANKS, make_requests, model_dir, plain_model
from infero_b200.config.dukolorn import DukolornConfig
from infero_b200.config.qwen2 import ConfigError
from infero_b200.models.decoder import DecoderModel
from infero_b200.parts.normed_attention import distance_buckets
from infero_b200.registry import load_config, resolve_architecture


def _spec(cfg):
    return DukolornConfig.from_dict(cfg).to_model_spec()


def test_the_registry_knows_the_name():
    assert resolve_architecture({"architecture": "Dukolorn"}).name == "Dukolorn"


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_fixture_reads_and_lowers(name):
    cfg = CONFIGS[name]
    spec = _spec(cfg)
    assert (spec.vocab_size, spec.hidden, spec.logit_scale) == (cfg["vocab"], cfg["width"], cfg["logit_scale"])
    assert not spec.tie_embeddings and spec.embed_norm.kind == "rmsnorm_centred" and spec.embed_norm_name == "embed.norm"
    assert [(e.block, e.cache) for e in spec.schedule] == [(i, i) for i in range(len(cfg["layers"]))]
    kinds = {"channel_delta": "channel_delta_memory", "parallel": "parallel", "latent_attention": "latent_attention"}
    for L, blk in zip(cfg["layers"], spec.blocks):
        assert blk.kind == "postnorm" and blk.mixer_norm.kind == "rmsnorm_centred" and blk.mixer_norm.eps == cfg["norm"]["eps"]
        assert blk.mixer.kind == kinds[L["type"]] and (blk.ffn is None) == (L["mlp"] is None)
        if blk.ffn is not None:
            assert (blk.ffn.kind, blk.ffn.intermediate, blk.ffn.bias) == ("swiglu", L["mlp"]["ff"], True)


def test_the_mixers_of_a_layer_list():
    par, lat, dl, _ = [b.mixer for b in _spec(CONFIGS["A"]).blocks]
    l, r = par.branches
    assert par.branch_scales == (0.7, 1.4) and not par.branch_norms
    assert (l.kind, l.num_heads, l.num_kv_heads, l.head_dim, l.v_dim, l.scale, l.distance_max) == ("normed_attention", 4, 2, 64, 64, 0.11, 60)
    assert (l.qk_norm_kind, l.softcap, l.q_temperature, l.sink_per_head, l.window) == ("projection", 6.0, (0.4, 32.0), True, None)
    assert l.position is None and not l.qkv_bias and dict(l.names)["sink"] == "mix.left.sink"
    assert (r.kind, r.num_heads, r.head_dim, r.v_dim, r.decay_tau) == ("decayed_memory", 2, 32, 48, 8.0)
    assert dict(r.names)["decay_bias"] == "mix.right.a2.b"
    assert (lat.num_heads, lat.head_dim, lat.rot_dim, lat.v_dim, lat.latent_dim, lat.scale, lat.window) == (4, 32, 16, 24, 64, 0.2, 39)
    assert (lat.position.kind, lat.position.theta, lat.position.rotary_dim, lat.sink_per_head) == ("rope_interleaved", 5000.0, 16, True)
    assert (dl.kind, dl.num_heads, dl.num_kv_heads, dl.head_dim, dl.v_dim, dl.conv_taps) == ("channel_delta_memory", 4, 2, 64, 32, 3)


def test_what_a_request_keeps():
    m = DecoderModel(_spec(CONFIGS["A"]))
    assert set(m.kv_specs) == {0, 1, 3} and set(m.state_specs) == {0, 2}
    assert (m.kv_specs[0].window, m.kv_specs[1].window, m.kv_specs[3].window) == (None, 39, 17)
    assert (m.kv_specs[1].num_kv_heads, m.kv_specs[1].head_dim, m.kv_specs[1].value_dim) == (1, 64 + 16, 0)
    assert m.state_specs[0].shape == (2 * 48 * 32,) and m.state_specs[0].dtype == torch.float32
    assert m.state_specs[2].shape == (2 * (2 * 2 * 64 + 4 * 32) + 4 * 32 * 64,)


def test_sizes_that_only_the_tensors_say():
    from infero_b200.weights.loader import load_tensors
    for name in ("A", "B"):
        mdir = model_dir(name)
        _, _, spec = load_config(mdir)
        model = DecoderModel(spec)
        t = load_tensors(mdir, model.declare(), "float32", "cpu")
        model.bind(t)
        for L, blk in zip(CONFIGS[name]["layers"], model.blocks):
            if L["type"] == "channel_delta":
                assert blk.mixer.ranks == {"decay_down": RANKS[name], "gate_down": RANKS[name] + 1}
                assert blk.mixer.input_rows()[0].shape[0] % 4 == 0
            if L["type"] == "parallel":
                a, b = blk.mixer.branches
                assert b.ranks == {"decay_down": RANKS[name]} and a.rel.shape[0] == L["mixer"]["left"]["heads"]
                rel, m = t[f"{blk.spec.prefix}.mix.left.rel"], L["mixer"]["left"]
                for n in (0, 1, 5, 40, 300):
                    row = PD.distance_bucket(n, BUCKETS[name], float(m["bias_max"]))
                    assert torch.equal(a.rel[:, min(n, a.rel.shape[1] - 1)], rel[row])
        # the logits' constant sits in the final norm's weight
        assert torch.allclose(model.final_norm.weight, (1 + t["final.norm"]) * CONFIGS[name]["logit_scale"])


def test_buckets_of_a_distance():
    for B, Dm in ((16, 120.0), (10, 60.0), (24, 12.5), (2, 2.0), (7, 90.0), (16, 128.0)):
        table = distance_buckets(B, Dm)
        for n in range(2 * int(Dm) + 5):
            got = table[min(n, len(table) - 1)]
            half = B // 2
            want = PD.distance_bucket(n, B, Dm)
            if got != want:                       # (a power that falls on a bucket's edge exactly: floating point may say one less)
                assert got == want + 1 and abs((n / half) ** (B - half) / (Dm / half) ** (got - half) - 1) < 1e-9


@pytest.mark.parametrize("path,value", [
    (("layers",), []), (("layers", 0, "type"), "attention"), (("norm", "eps"), 0), (("vocab",), 1.5),
    (("layers", 0, "mixer", "left", "kv_heads"), 3), (("layers", 0, "mixer", "left", "softcap"), -1.0),
    (("layers", 0, "mixer", "left", "q_temp", "every"), 0), (("layers", 0, "mixer", "left_scale"), "1"),
    (("layers", 0, "mixer", "right", "tau"), 0), (("layers", 1, "mixer", "rot", "dims"), 18), (("layers", 1, "mixer", "rot", "dims"), 3),
    (("layers", 1, "mixer", "mask", "size"), 0), (("layers", 1, "mixer", "kv_rank"), None), (("layers", 2, "mixer", "conv"), 17),
    (("layers", 0, "mlp", "kind"), "moe"), (("layers", 0, "mlp", "ff"), 0)])
def test_what_is_refused(path, value):
    cfg = copy.deepcopy(CONFIGS["A"])
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        _spec(cfg)


def test_what_may_be_absent():
    cfg = copy.deepcopy(CONFIGS["A"])
    del cfg["logit_scale"], cfg["layers"][0]["mixer"]["left"]["q_temp"], cfg["layers"][0]["mixer"]["left"]["softcap"]
    del cfg["layers"][1]["mixer"]["mask"]
    spec = _spec(cfg)
    l = spec.blocks[0].mixer.branches[0]
    assert spec.logit_scale == 1.0 and l.q_temperature is None and l.softcap == 0 and spec.blocks[1].mixer.window is None


def test_the_plain_statement_sees_what_the_fixtures_stress():
    """In the fixtures a window that is one off, a missing sink, a missing temperature, a wrong cap or lost decays move the
    logits by far more than the tolerances."""
    cfg, w = plain_model(model_dir("A"))
    toks = make_requests("A", [90], seed=3)["r0"]
    base = PD.forward(cfg, w, toks)

    def moved(c=cfg, ww=w):
        return float((PD.forward(c, ww, toks) - base).abs().max() / base.abs().max())
    for path, value in ((("layers", 1, "mixer", "mask", "size"), 38), (("layers", 0, "mixer", "left", "q_temp", "coef"), 0.0),
                        (("layers", 0, "mixer", "left", "softcap"), 30.0), (("layers", 0, "mixer", "right", "tau"), 9.0)):
        c = copy.deepcopy(cfg)
        at = c
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        assert moved(c) > 1e-3, path
    for k in ("l0.mix.left.sink", "l1.mix.sink"):
        assert moved(ww={**w, k: w[k] - 50.0}) > 1e-2, k
    assert moved(ww={**w, "l2.mix.dt_bias": w["l2.mix.dt_bias"] + 5.0}) > 1e-2


