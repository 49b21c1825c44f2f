"""The Puresun decoder as a :class:`ModelSpec`.

A stack of blocks whose two sublayers read the output of one RMS norm side by side, ``x <- x + (mixer(h) + ff(h))``.
A table of rows by hashed token pairs joins the token embedding (the previous token is part of a request's
state).  The mixer is latent attention with a rotated key part (half-split rotation), a sliding window and a
sigmoid gate per channel; the feed-forward is a mixture of ungated experts, ``W_down relu(W_up h)^2``, with a
softmax router whose weights are taken over the chosen experts only; a layer may lack it.  A span of the layers
may run several times in a row with the same weights and a cache of its own per pass: before every pass a vector
of the pass joins the stream, before every pass but the first the embedded rows do once more.  The head is
untied, the logits are capped.

    {"architecture": "Puresun", "vocab": V, "width": W, "norm": {"eps": e}, "logit_softcap": cap,
     "embedding": {"bigram": {"buckets": B, "mul_prev": a, "mul_cur": b}},
     "loop": {"start": i, "stop": j, "times": n},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot": {"base", "dims"}, "mask": {"size"}},
                 "mlp": {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}} | null}, ...]}

Tensors are ``embed``, ``bigram``, ``loop.step``, ``head``, ``final.norm`` and, for layer ``i``, ``l<i>.norm1``,
``l<i>.mix.*`` and, with a feed-forward, ``l<i>.mlp.router`` and ``l<i>.mlp.e<k>.{up,down}``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from ..config.model_config import ConfigError
from ..parts.block import ParallelBlockSpec
from ..parts.embedding import BigramEmbeddingSpec, EmbeddingSpec, HeadSpec
from ..parts.feedforward import MoESpec
from ..parts.latent import LatentAttentionSpec
from ..parts.norm import RMSNormSpec
from ..parts.position import NoPositionSpec, RopeHalvesSpec
from .decoder import LayerCall, ModelSpec, StreamInput

ARCHITECTURE = "Puresun"
DEFAULT_MAX_POSITIONS = 1 << 17     # the design has no limit of its own
LOOP_TABLE = "loop.step"


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LatentLayer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class MoELayer:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class PuresunLayer:
    type: str                      # "latent_attention"
    mixer: LatentLayer
    mlp: MoELayer | None


@dataclass(frozen=True)
class PuresunConfig:
    """Typed configuration; the first four fields are what the engine reads."""

    architecture: str
    vocab_size: int
    max_position_embeddings: int
    eos_token_ids: tuple
    hidden_size: int
    norm_eps: float
    bigram: Bigram | None
    loop: tuple | None             # (start, stop, times)
    logit_softcap: float | None
    layers: tuple


def _need(raw: Mapping[str, Any], key: str, where: str) -> Any:
    if not isinstance(raw, Mapping) or key not in raw or raw[key] is None:
        raise ConfigError(f"config.json is missing {where}{key!r}")
    return raw[key]


def _integer(value: Any, what: str, least: int = 1) -> int:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or int(value) != value or int(value) < least:
        raise ConfigError(f"{what} must be an integer of at least {least}, got {value!r}")
    return int(value)


def _number(value: Any, what: str) -> float:
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ConfigError(f"{what} must be a number, got {value!r}")
    return float(value)


def _parse_mixer(m: Mapping[str, Any], w: str) -> LatentLayer:
    num = lambda key: _integer(_need(m, key, w), w + key)
    rot_dim = _integer(m.get("rot_dim") or 0, w + "rot_dim", 0)
    dims, base = 0, 1.0
    if rot_dim:
        rot = _need(m, "rot", w)
        dims = _integer(rot.get("dims", rot_dim), w + "rot.dims", 0)
        if dims % 2 or dims > rot_dim:
            raise ConfigError(f"{w}rot.dims must be even and at most rot_dim ({rot_dim}), got {dims}")
        base = _number(_need(rot, "base", w + "rot."), w + "rot.base")
        if not base > 0.0:
            raise ConfigError(f"{w}rot.base must be > 0, got {base}")
    dim = num("dim")
    return LatentLayer(heads=num("heads"), dim=dim, rot_dim=rot_dim, vdim=_integer(m.get("vdim", dim), w + "vdim"),
                       kv_rank=num("kv_rank"), scale=_number(_need(m, "scale", w), w + "scale"),
                       window=_integer(_need(_need(m, "mask", w), "size", w + "mask."), w + "mask.size"),
                       rot_dims=dims, rot_base=base)


def _parse_mlp(raw: Any, where: str) -> MoELayer | None:
    if raw is None:
        return None
    if raw.get("kind", "moe") != "moe":
        raise ConfigError(f"{where}kind {raw.get('kind')!r} is not a feed-forward of this design (moe)")
    router, w = _need(raw, "router", where), where + "router."
    experts, top = _integer(_need(router, "experts", w), w + "experts"), _integer(_need(router, "top", w), w + "top")
    if top > experts:
        raise ConfigError(f"{w}top ({top}) is more than the number of experts ({experts})")
    return MoELayer(ff=_integer(_need(_need(raw, "expert", where), "ff", where + "expert."), where + "expert.ff"),
                    experts=experts, top=top)


def _parse_layer(i: int, raw: Mapping[str, Any]) -> PuresunLayer:
    where = f"layers[{i}]."
    kind = _need(raw, "type", where)
    if kind != "latent_attention":
        raise ConfigError(f"{where}type {kind!r} is not a mixer of this design (latent_attention)")
    return PuresunLayer(type=kind, mixer=_parse_mixer(_need(raw, "mixer", where), where + "mixer."),
                        mlp=_parse_mlp(raw.get("mlp"), where + "mlp."))


def _parse_loop(loop: Any, n: int) -> tuple | None:
    if loop is None:
        return None
    start, stop = (_integer(_need(loop, k, "loop."), f"loop.{k}", 0) for k in ("start", "stop"))
    if not start < stop <= n:
        raise ConfigError(f"loop.start ({start}) and loop.stop ({stop}) do not name a span of the {n} layers")
    return start, stop, _integer(_need(loop, "times", "loop."), "loop.times")


def parse_config(raw: Mapping[str, Any], eos_token_ids=None) -> PuresunConfig:
    """The typed configuration of a ``config.json`` dictionary."""
    layers_raw = _need(raw, "layers", "")
    if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
        raise ConfigError("config.json: layers must be a non-empty list")
    eps = _number(_need(_need(raw, "norm", ""), "eps", "norm."), "norm.eps")
    if not eps > 0.0:
        raise ConfigError(f"norm.eps must be > 0, got {eps}")
    bigram = (raw.get("embedding") or {}).get("bigram")
    if bigram is not None:
        w = "embedding.bigram."
        bigram = Bigram(buckets=_integer(_need(bigram, "buckets", w), w + "buckets"),
                        mul_prev=_integer(_need(bigram, "mul_prev", w), w + "mul_prev", 0),
                        mul_cur=_integer(_need(bigram, "mul_cur", w), w + "mul_cur", 0))
    cap = raw.get("logit_softcap")
    if cap is not None and not _number(cap, "logit_softcap") > 0.0:
        raise ConfigError(f"logit_softcap must be > 0, got {cap}")
    return PuresunConfig(
        architecture=ARCHITECTURE,
        vocab_size=_integer(_need(raw, "vocab", ""), "vocab"),
        max_position_embeddings=_integer(raw.get("max_position_embeddings", DEFAULT_MAX_POSITIONS),
                                         "max_position_embeddings"),
        eos_token_ids=tuple(int(e) for e in (eos_token_ids or ())),
        hidden_size=_integer(_need(raw, "width", ""), "width"),
        norm_eps=eps,
        bigram=bigram,
        loop=_parse_loop(raw.get("loop"), len(layers_raw)),
        logit_softcap=None if cap is None else float(cap),
        layers=tuple(_parse_layer(i, lay) for i, lay in enumerate(layers_raw)),
    )


def schedule_of(cfg: PuresunConfig) -> tuple:
    """The calls in the order in which they run: the layers before the looped span, the span ``times`` times, each
    pass with caches of its own and with its vector (and, from the second pass on, the embedded rows) joining the
    stream in front of its first layer, then the rest."""
    n = len(cfg.layers)
    start, stop, times = cfg.loop or (n, n, 0)
    calls = [LayerCall(f"l{i}", f"l{i}") for i in range(start)]
    for t in range(times):
        for i in range(start, stop):
            joins = StreamInput(embedding=t > 0, table=LOOP_TABLE, row=t) if i == start else None
            calls.append(LayerCall(f"l{i}", f"l{i}" if t == 0 else f"l{i}.pass{t}", joins))
    return tuple(calls + [LayerCall(f"l{i}", f"l{i}") for i in range(stop, n)])


def model_spec(cfg: PuresunConfig) -> ModelSpec:
    """Blocks and schedule: a block per layer; a layer of the looped span is called once per pass."""
    width, eps = cfg.hidden_size, cfg.norm_eps
    norm = RMSNormSpec(width, eps)
    blocks = []
    for i, lay in enumerate(cfg.layers):
        prefix = f"l{i}."
        m, ffn = lay.mixer, {}
        position = RopeHalvesSpec(m.rot_dims, m.rot_base) if m.rot_dims else NoPositionSpec()
        mixer = LatentAttentionSpec(hidden_size=width, num_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim,
                                    kv_rank=m.kv_rank, softmax_scale=m.scale, norm_eps=eps, rot_dim=m.rot_dim,
                                    position=position, window=m.window, gate=True)
        if lay.mlp is not None:
            f = lay.mlp
            ffn = dict(feed_forward=MoESpec(hidden_size=width, intermediate_size=f.ff, num_experts=f.experts, top=f.top,
                                            correction=False, gated=False, router="softmax", activation="relu2"),
                       ffn_prefix=prefix + "mlp.")
        blocks.append(ParallelBlockSpec(name=f"l{i}", norm1=norm, mixer=mixer, norm1_name=prefix + "norm1",
                                        mixer_prefix=prefix + "mix.", **ffn))
    b = cfg.bigram
    return ModelSpec(
        embedding=(EmbeddingSpec(cfg.vocab_size, width, name="embed") if b is None else
                   BigramEmbeddingSpec(cfg.vocab_size, width, b.buckets, b.mul_prev, b.mul_cur)),
        blocks=tuple(blocks),
        schedule=schedule_of(cfg),
        final_norm=norm,
        final_norm_name="final.norm",
        head=HeadSpec(cfg.vocab_size, width, tied=False, name="head", softcap=cfg.logit_softcap),
        stream_tables=((LOOP_TABLE, cfg.loop[2]),) if cfg.loop is not None else (),
    )
