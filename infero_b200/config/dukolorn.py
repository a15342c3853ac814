"""Typed configuration of the Dukolorn decoder, read from its own config.json keys.

config.json: ``architecture`` "Dukolorn", ``vocab``, ``width``, ``norm.eps``, ``logit_scale`` and ``layers``.  Layer i's tensors
start with ``l<i>.``; an entry gives ``type``, ``mixer`` and ``mlp`` (null, or {``kind`` "dense", ``ff``}: a SwiGLU whose
projections have biases).  The sublayers read the residual stream itself and an RMS norm sits on each one's result, its
weight stored as the distance from one; the embedding and the output product's input have such norms too.

``type`` "channel_delta": the gated delta rule with a decay per key channel (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``
taps).

``type`` "parallel": two mixers side by side on the same input, ``mixer.left`` and ``mixer.right``, added up with
``left_scale`` and ``right_scale``.  Left: causal grouped-query attention (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``) with
norms over the whole query and key projections, a temperature of the queries that grows with the position (``q_temp``
{``coef``, ``every``}), soft-capped scores (``softcap``), a learned bias by distance up to ``bias_max`` (its table says how many
buckets) and a learned sink per head.  Right: gated linear attention (``heads``, ``dim``, ``vdim``, ``tau``).

``type`` "latent_attention": latent attention (``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``rot`` {``base``,
``dims``}) over a sliding window (``mask.size``), with a learned sink per head.

The widths of the narrow middles (``.a1``, ``.g1``) and the rows of the distance tables are the stored tensors' own.

Lowering: blocks "postnorm"; mixers "channel_delta_memory", "latent_attention", and "parallel" over "normed_attention" and
"decayed_memory"; feed-forward "swiglu" with biases; a norm of the embedding.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .gositar import _number
from .nuvarax import _grouped_heads, _object, _taps
from .qwen2 import ConfigError
from .spec import (BlockSpec, DECAYED_MEMORY_NAMES, FeedForwardSpec, MixerSpec, ModelSpec, NormSpec, NORMED_ATTENTION_NAMES,
                   PositionSpec, ScheduleEntry)
from .vufizen import _pos_int

RANDOM_BUCKETS = 32              # buckets of the distance table where weights are made, not loaded
RANDOM_RANK = 64                 # width of the narrow middles there


@dataclass(frozen=True)
class DukolornDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class DukolornLeft:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    softcap: float                             # 0: scores as they are
    q_temp: Optional[Tuple[float, float]]      # coef, every


@dataclass(frozen=True)
class DukolornRight:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class DukolornLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_dims: int
    rot_base: float
    window: Optional[int]


@dataclass(frozen=True)
class DukolornLayer:
    type: str                                  # "channel_delta" | "parallel" | "latent_attention"
    delta: Optional[DukolornDelta] = None
    left: Optional[DukolornLeft] = None
    right: Optional[DukolornRight] = None
    scales: Tuple[float, float] = (1.0, 1.0)
    latent: Optional[DukolornLatent] = None
    ff: int = 0                                # 0: no feed-forward


def _left(m: Dict[str, Any], where: str) -> DukolornLeft:
    temp = None
    if m.get("q_temp") is not None:
        t = _object(m, "q_temp", where + ".")
        temp = (_number(t, "coef", where + ".q_temp", positive=False), _number(t, "every", where + ".q_temp"))
    cap = _number(m, "softcap", where) if m.get("softcap") is not None else 0.0
    return DukolornLeft(*_grouped_heads(m, where), _number(m, "scale", where, positive=False), _number(m, "bias_max", where), cap, temp)


def _latent(m: Dict[str, Any], where: str) -> DukolornLatent:
    heads, dim, vdim, rank = (_pos_int(m, k, where) for k in ("heads", "dim", "vdim", "kv_rank"))
    rot_dim = m.get("rot_dim")
    if isinstance(rot_dim, bool) or not isinstance(rot_dim, int) or rot_dim < 0:
        raise ConfigError(f"config.json: {where}.rot_dim must be an integer of at least 0, got {rot_dim!r}")
    dims, base = 0, 10000.0
    if rot_dim:
        rot = _object(m, "rot", where + ".")
        dims, base = _pos_int(rot, "dims", where + ".rot"), _number(rot, "base", where + ".rot")
        if dims % 2 or dims > rot_dim:
            raise ConfigError(f"config.json: {where}.rot.dims {dims} is odd or beyond rot_dim {rot_dim}")
    window = _pos_int(_object(m, "mask", where + "."), "size", where + ".mask") if m.get("mask") is not None else None
    return DukolornLatent(heads, dim, rot_dim, vdim, rank, _number(m, "scale", where, positive=False), dims, base, window)


def _layer(L: Any, where: str) -> DukolornLayer:
    if not isinstance(L, dict):
        raise ConfigError(f"config.json: {where} is not an object")
    m, wm, ff = _object(L, "mixer", where + "."), where + ".mixer", 0
    if L.get("mlp") is not None:
        mlp = _object(L, "mlp", where + ".")
        if mlp.get("kind") != "dense":
            raise ConfigError(f"config.json: {where}.mlp.kind {mlp.get('kind')!r} is not 'dense'")
        ff = _pos_int(mlp, "ff", where + ".mlp")
    kind = L.get("type")
    if kind == "channel_delta":
        return DukolornLayer(kind, delta=DukolornDelta(*_grouped_heads(m, wm), _taps(m, "conv", wm)), ff=ff)
    if kind == "latent_attention":
        return DukolornLayer(kind, latent=_latent(m, wm), ff=ff)
    if kind == "parallel":
        r, wr = _object(m, "right", wm + "."), wm + ".right"
        right = DukolornRight(_pos_int(r, "heads", wr), _pos_int(r, "dim", wr), _pos_int(r, "vdim", wr), _number(r, "tau", wr))
        scales = tuple(_number(m, k, wm, positive=False) for k in ("left_scale", "right_scale"))
        return DukolornLayer(kind, left=_left(_object(m, "left", wm + "."), wm + ".left"), right=right, scales=scales, ff=ff)
    raise ConfigError(f"config.json: {where}.type {kind!r} is none of 'channel_delta', 'parallel', 'latent_attention'")


@dataclass(frozen=True)
class DukolornConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    layers: Tuple[DukolornLayer, ...]
    raw: Tuple[Tuple[str, Any], ...] = ()

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "DukolornConfig":
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        scale = _number(raw, "logit_scale", "config", positive=False) if raw.get("logit_scale") is not None else 1.0
        return cls(_pos_int(raw, "vocab", "config"), _pos_int(raw, "width", "config"), _number(raw.get("norm") or {}, "eps", "norm"), scale,
                   tuple(_layer(L, f"layers[{i}]") for i, L in enumerate(entries)), raw=tuple(raw.items()))

    def to_json_dict(self) -> Dict[str, Any]:
        return {k: v for k, v in self.raw if k in ("architecture", "vocab", "width", "norm", "logit_scale", "layers")}

    # ---- lowering to parts ---------------------------------------------------------------------
    def _mixer(self, L: DukolornLayer) -> MixerSpec:
        d = self.width
        if L.type == "channel_delta":
            m = L.delta
            return MixerSpec(kind="channel_delta_memory", hidden=d, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim,
                             value_dim=m.vdim, conv_taps=m.conv, norm_eps=self.eps, low_rank=RANDOM_RANK, weight_suffix="")
        if L.type == "latent_attention":
            m = L.latent
            rot = PositionSpec("rope_interleaved", m.rot_base, m.rot_dims) if m.rot_dims else None
            return MixerSpec(kind="latent_attention", hidden=d, num_heads=m.heads, num_kv_heads=1, head_dim=m.dim, rot_dim=m.rot_dim,
                             value_dim=m.vdim, latent_dim=m.kv_rank, scale=m.scale, position=rot, window=m.window, sink_per_head=True,
                             norm_eps=self.eps, weight_suffix="")
        rename = lambda table, side: tuple((r, leaf.replace("mix.", f"mix.{side}.", 1)) for r, leaf in table)   # noqa: E731
        a, r = L.left, L.right
        left = MixerSpec(kind="normed_attention", hidden=d, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, value_dim=a.vdim,
                         scale=a.scale, qk_norm_kind="projection", q_temperature=a.q_temp, softcap=a.softcap,
                         distance_buckets=RANDOM_BUCKETS, distance_max=a.bias_max, sink_per_head=True, scale_values=True,
                         norm_eps=self.eps, names=rename(NORMED_ATTENTION_NAMES, "left"), weight_suffix="")
        right = MixerSpec(kind="decayed_memory", hidden=d, num_heads=r.heads, head_dim=r.dim, value_dim=r.vdim, decay_tau=r.tau,
                          low_rank=RANDOM_RANK, norm_eps=self.eps, names=rename(DECAYED_MEMORY_NAMES, "right"), weight_suffix="")
        return MixerSpec(kind="parallel", hidden=d, branches=(left, right), branch_scales=L.scales, norm_eps=self.eps, weight_suffix="")

    def to_model_spec(self) -> ModelSpec:
        norm = NormSpec(kind="rmsnorm_centred", dim=self.width, eps=self.eps)
        blocks = []
        for i, L in enumerate(self.layers):
            ffn = None
            if L.ff:
                ffn = FeedForwardSpec(kind="swiglu", hidden=self.width, intermediate=L.ff, bias=True, weight_suffix="",
                                      names=(("gate", "mlp.gate"), ("up", "mlp.up"), ("down", "mlp.down")))
            blocks.append(BlockSpec(kind="postnorm", prefix=f"l{i}", mixer=self._mixer(L), ffn=ffn, mixer_norm=norm,
                                    ffn_norm=norm if ffn is not None else None, mixer_norm_name="norm1", ffn_norm_name="norm2"))
        return ModelSpec(architecture="Dukolorn", vocab_size=self.vocab, hidden=self.width, blocks=tuple(blocks),
                         schedule=tuple(ScheduleEntry(block=i, cache=i) for i in range(len(blocks))), final_norm=norm,
                         tie_embeddings=False, embed_name="embed", final_norm_name="final.norm", head_name="head",
                         logit_scale=self.logit_scale, embed_norm=norm, embed_norm_name="embed.norm")
