"""The Sofinex decoder as a :class:`ModelSpec`.

A stack of pre-norm blocks with RMS norms whose weights are stored around zero; a span of the layers may run several
times in a row with the same weights and a cache or state of its own per pass.  The mixers, listed layer by layer
in ``config.json``:

* ``attention``: differential attention (two maps per head over the same values, the second subtracted), half-split
  rotation stretched by wavelength, a sliding window.
* ``parallel``: two mixers side by side, half the sum of their outputs, each normed over the model's width.  Left:
  grouped-query attention with YaRN-stretched half-split rotation, q and k divided by their root mean square after
  it, a sliding window and a sink per head.  Right: the gated delta rule with a decay per key channel, decay and
  output gate from low-rank projections.

Feed-forwards are dense with the exact gelu or mixtures of silu-gated experts with a softmax router, identity
experts among the router's outputs and a gated shared expert; a layer may lack its feed-forward.  The embedding is
scaled, the head untied.

    {"architecture": "Sofinex", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "loop": {"start": i, "stop": j, "times": n},
     "layers": [{"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "diff", "mask": {"size"},
                                                "rot": {"base", "dims", "scaling": {"factor", "low", "high", "original"}}},
                 "mlp": ...},
                {"type": "parallel", "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"},
                                                        "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}},
                                               "right": {"heads", "kv_heads", "dim", "vdim", "conv"}}, "mlp": ...}, ...]}
    mlp: {"kind": "dense", "ff": F}
       | {"kind": "moe", "expert": {"ff"}, "shared": {"ff"},
          "router": {"experts", "identity", "top", "groups": {"count", "keep"}}} | null

Tensors are ``embed``, ``head``, ``final.norm`` and, for layer ``i``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` (for a
parallel layer ``l<i>.mix.left.*`` and ``l<i>.mix.right.*``) and ``l<i>.mlp.*``.  The ranks of a right half's low-rank
projections are the row counts of its ``a1`` and ``g1``: they are read from the checkpoint's header or, for a folder of
random weights, from the optional keys ``right.decay_rank`` and ``right.gate_rank``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from ..config.model_config import ConfigError
from ..parts.attention import GatedAttentionSpec
from ..parts.block import PreNormBlockSpec
from ..parts.delta import GatedDeltaSpec
from ..parts.differential import DifferentialAttentionSpec
from ..parts.embedding import EmbeddingSpec, HeadSpec
from ..parts.feedforward import MlpSpec, MoESpec
from ..parts.norm import OffsetRMSNormSpec
from ..parts.parallel import ParallelMixerSpec
from ..parts.position import NoPositionSpec, RopeHalvesSpec, WaveScaling, YarnScaling
from .decoder import LayerCall, ModelSpec

ARCHITECTURE = "Sofinex"
DEFAULT_MAX_POSITIONS = 1 << 17     # the design has no limit of its own
DEFAULT_RANK = 16                   # of the low-rank projections, where neither checkpoint nor configuration gives it
UNIT_EPS = 1e-6                     # under the root when q and k of the delta rule are scaled to unit length
HALF = 0.5                          # the factor on either half of a parallel mixer


@dataclass(frozen=True)
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    position: object
    diff: float | None = None


@dataclass(frozen=True)
class DeltaSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int
    gate_rank: int


@dataclass(frozen=True)
class ParallelLayer:
    left: AttentionSizes
    right: DeltaSizes


@dataclass(frozen=True)
class DenseLayer:
    ff: int


@dataclass(frozen=True)
class MoELayer:
    ff: int
    experts: int
    identity: int
    top: int
    groups: int
    keep: int
    shared_ff: int | None


@dataclass(frozen=True)
class SofinexLayer:
    type: str                      # "attention" or "parallel"
    mixer: Any
    mlp: Any                       # DenseLayer, MoELayer or None


@dataclass(frozen=True)
class SofinexConfig:
    """Typed configuration; the first four fields are what the engine reads."""

    architecture: str
    vocab_size: int
    max_position_embeddings: int
    eos_token_ids: tuple
    hidden_size: int
    norm_eps: float
    embedding_scale: float
    loop: tuple                    # (start, stop, times)
    layers: tuple


def _need(raw: Mapping[str, Any], key: str, where: str) -> Any:
    if not isinstance(raw, Mapping) or key not in raw or raw[key] is None:
        raise ConfigError(f"config.json is missing {where}{key!r}")
    return raw[key]


def _integer(value: Any, what: str, least: int = 1) -> int:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or int(value) != value or int(value) < least:
        raise ConfigError(f"{what} must be an integer of at least {least}, got {value!r}")
    return int(value)


def _number(value: Any, what: str, above: float | None = None) -> float:
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ConfigError(f"{what} must be a number, got {value!r}")
    if above is not None and not value > above:
        raise ConfigError(f"{what} must be > {above:g}, got {value!r}")
    return float(value)


def _parse_position(rot: Any, dim: int, w: str, kind, keys: tuple):
    """The half-split rotation of ``rot``; ``kind`` is the class of its scaling and ``keys`` that class's fields."""
    if rot is None:
        return NoPositionSpec()
    dims = _integer(rot.get("dims", dim), w + "dims", 0)
    if dims % 2 or dims > dim:
        raise ConfigError(f"{w}dims must be an even number up to the head size {dim}, got {dims}")
    if dims == 0:
        return NoPositionSpec()
    base = _number(_need(rot, "base", w), w + "base", above=0.0)
    scaling = rot.get("scaling")
    if scaling is not None:
        ws = w + "scaling."
        scaling = kind(**{key: _number(_need(scaling, key, ws), ws + key, above=0.0) for key in keys})
        if isinstance(scaling, WaveScaling) and scaling.high < scaling.low:
            raise ConfigError(f"{ws}high ({scaling.high:g}) lies below low ({scaling.low:g})")
        if isinstance(scaling, YarnScaling) and not base > 1.0:
            raise ConfigError(f"{w}base must be > 1 for this scaling, got {base:g}")
    return RopeHalvesSpec(dims, base, scaling=scaling)


def _parse_heads(m: Mapping[str, Any], w: str) -> dict:
    heads = _integer(_need(m, "heads", w), w + "heads")
    kv = _integer(m.get("kv_heads", heads), w + "kv_heads")
    if heads % kv:
        raise ConfigError(f"{w}heads ({heads}) must be a multiple of kv_heads ({kv})")
    dim = _integer(_need(m, "dim", w), w + "dim")
    return dict(heads=heads, kv_heads=kv, dim=dim, vdim=_integer(m.get("vdim", dim), w + "vdim"))


def _parse_attention(m: Mapping[str, Any], w: str, differential: bool) -> AttentionSizes:
    sizes = _parse_heads(m, w)
    kind, keys = ((WaveScaling, ("factor", "original", "low", "high")) if differential else
                  (YarnScaling, ("factor", "original", "fast", "slow")))
    diff = _number(_need(m, "diff", w), w + "diff") if differential else None
    return AttentionSizes(**sizes, scale=_number(_need(m, "scale", w), w + "scale"),
                          window=_integer(_need(_need(m, "mask", w), "size", w + "mask."), w + "mask.size"),
                          position=_parse_position(m.get("rot"), sizes["dim"], w + "rot.", kind, keys), diff=diff)


def _parse_mlp(raw: Any, where: str):
    if raw is None:
        return None
    kind = _need(raw, "kind", where)
    if kind == "dense":
        return DenseLayer(_integer(_need(raw, "ff", where), where + "ff"))
    if kind != "moe":
        raise ConfigError(f"{where}kind {kind!r} is not a feed-forward of this design (dense, moe)")
    router, w = _need(raw, "router", where), where + "router."
    experts, top = _integer(_need(router, "experts", w), w + "experts"), _integer(_need(router, "top", w), w + "top")
    identity = _integer(router.get("identity") or 0, w + "identity", 0)
    groups = router.get("groups") or {}
    count = _integer(groups.get("count", 1), w + "groups.count")
    keep = _integer(groups.get("keep", count), w + "groups.keep")
    total = experts + identity
    if total % count or keep > count:
        raise ConfigError(f"{w}{total} outputs do not form {count} equal groups of which {keep} are kept")
    if top > keep * (total // count):
        raise ConfigError(f"{w}top ({top}) is more than the {keep} kept groups of {total // count} outputs hold")
    shared = raw.get("shared")
    return MoELayer(ff=_integer(_need(_need(raw, "expert", where), "ff", where + "expert."), where + "expert.ff"),
                    experts=experts, identity=identity, top=top, groups=count, keep=keep,
                    shared_ff=None if shared is None else _integer(_need(shared, "ff", where + "shared."), where + "shared.ff"))


def _parse_layer(i: int, raw: Mapping[str, Any], shapes: Mapping[str, tuple]) -> SofinexLayer:
    where = f"layers[{i}]."
    kind, m, w = _need(raw, "type", where), _need(raw, "mixer", where), where + "mixer."
    if kind == "attention":
        mixer = _parse_attention(m, w, differential=True)
    elif kind == "parallel":
        r, wr = _need(m, "right", w), w + "right."
        ranks = {}
        for key, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
            shape = shapes.get(f"l{i}.mix.right.{name}")
            rank = shape[0] if shape is not None and len(shape) == 2 else r.get(key, DEFAULT_RANK)
            ranks[key] = _integer(rank, wr + key)
        mixer = ParallelLayer(left=_parse_attention(_need(m, "left", w), w + "left.", differential=False),
                              right=DeltaSizes(**_parse_heads(r, wr), conv=_integer(_need(r, "conv", wr), wr + "conv"), **ranks))
    else:
        raise ConfigError(f"{where}type {kind!r} is not a mixer of this design (attention, parallel)")
    return SofinexLayer(type=kind, mixer=mixer, mlp=_parse_mlp(raw.get("mlp"), where + "mlp."))


def _parse_loop(loop: Any, n: int) -> tuple:
    if loop is None:
        return 0, 0, 1
    start, stop = (_integer(_need(loop, k, "loop."), f"loop.{k}", 0) for k in ("start", "stop"))
    if not start <= stop <= n:
        raise ConfigError(f"loop.start ({start}) and loop.stop ({stop}) do not name a span of the {n} layers")
    return start, stop, _integer(_need(loop, "times", "loop."), "loop.times")


def parse_config(raw: Mapping[str, Any], eos_token_ids=None, tensor_shapes: Mapping[str, tuple] | None = None
                 ) -> SofinexConfig:
    """The typed configuration of a ``config.json`` dictionary.  ``tensor_shapes`` (name -> shape, from the
    checkpoint's header) supplies the ranks of the low-rank projections."""
    layers_raw = _need(raw, "layers", "")
    if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
        raise ConfigError("config.json: layers must be a non-empty list")
    return SofinexConfig(
        architecture=ARCHITECTURE,
        vocab_size=_integer(_need(raw, "vocab", ""), "vocab"),
        max_position_embeddings=_integer(raw.get("max_position_embeddings", DEFAULT_MAX_POSITIONS),
                                         "max_position_embeddings"),
        eos_token_ids=tuple(int(e) for e in (eos_token_ids or ())),
        hidden_size=_integer(_need(raw, "width", ""), "width"),
        norm_eps=_number(_need(_need(raw, "norm", ""), "eps", "norm."), "norm.eps", above=0.0),
        embedding_scale=_number((raw.get("embedding") or {}).get("scale", 1.0), "embedding.scale"),
        loop=_parse_loop(raw.get("loop"), len(layers_raw)),
        layers=tuple(_parse_layer(i, lay, tensor_shapes or {}) for i, lay in enumerate(layers_raw)),
    )


def schedule_of(cfg: SofinexConfig) -> tuple:
    """The calls in the order in which they run: the layers before the looped span, the span ``times`` times with
    caches of its own per pass, the rest."""
    start, stop, times = cfg.loop
    order = [(i, 0) for i in range(start)] + [(i, p) for p in range(times) for i in range(start, stop)]
    order += [(i, 0) for i in range(stop, len(cfg.layers))]
    return tuple(LayerCall(f"l{i}", f"l{i}" if p == 0 else f"l{i}.pass{p}") for i, p in order)


def _mixer_spec(m, width: int, eps: float):
    if isinstance(m, AttentionSizes):
        return DifferentialAttentionSpec(hidden_size=width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim,
                                         v_head_dim=m.vdim, softmax_scale=m.scale, position=m.position, diff=m.diff,
                                         norm_eps=eps, window=m.window)
    l, r = m.left, m.right
    left = GatedAttentionSpec(hidden_size=width, num_heads=l.heads, num_kv_heads=l.kv_heads, head_dim=l.dim,
                              v_head_dim=l.vdim, softmax_scale=l.scale, position=l.position, head_norm_eps=eps,
                              head_norm_weight=False, norm_after=True, sinks=True, window=l.window, pad_rows=True)
    right = GatedDeltaSpec(hidden_size=width, num_heads=r.heads, num_kv_heads=r.kv_heads, key_dim=r.dim,
                           value_dim=r.vdim, conv_taps=r.conv, norm_eps=eps, unit_eps=UNIT_EPS, decay_rank=r.decay_rank,
                           gate_rank=r.gate_rank, gate="sigmoid")
    return ParallelMixerSpec(left=left, right=right, left_scale=HALF, right_scale=HALF, out_norm_eps=eps)


def _feed_forward_spec(f, width: int):
    if isinstance(f, DenseLayer):
        return MlpSpec(width, f.ff, activation="gelu")
    return MoESpec(hidden_size=width, intermediate_size=f.ff, num_experts=f.experts, top=f.top, num_groups=f.groups,
                   keep_groups=f.keep, router="softmax_all", normalize=True, group_score="best", identity=f.identity,
                   shared_size=f.shared_ff, pad_inner=True)


def model_spec(cfg: SofinexConfig) -> ModelSpec:
    """Blocks and schedule: a block per layer; a layer of the looped span is called once per pass, each call with
    caches of its own (pages for attention, a state record for the delta rule)."""
    width, eps = cfg.hidden_size, cfg.norm_eps
    norm = OffsetRMSNormSpec(width, eps)
    blocks = []
    for i, lay in enumerate(cfg.layers):
        prefix = f"l{i}."
        ffn = dict(norm2=None, feed_forward=None, norm2_name=None, ffn_prefix=None)
        if lay.mlp is not None:
            ffn = dict(norm2=norm, feed_forward=_feed_forward_spec(lay.mlp, width), norm2_name=prefix + "norm2",
                       ffn_prefix=prefix + "mlp.")
        blocks.append(PreNormBlockSpec(name=f"l{i}", norm1=norm, mixer=_mixer_spec(lay.mixer, width, eps),
                                       norm1_name=prefix + "norm1", mixer_prefix=prefix + "mix.", **ffn))
    return ModelSpec(
        embedding=EmbeddingSpec(cfg.vocab_size, width, name="embed", scale=cfg.embedding_scale),
        blocks=tuple(blocks),
        schedule=schedule_of(cfg),
        final_norm=norm,
        final_norm_name="final.norm",
        head=HeadSpec(cfg.vocab_size, width, tied=False, name="head"),
    )
