"""Token embedding and the output head."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ..cache.manager import StateNeed
from ..csrc import ops
from .base import EMBEDDINGS, HEADS, Runtime, TensorReq, chain_of, linear, sum_parts, tensor_bytes


@dataclass(frozen=True)
class EmbeddingSpec:
    vocab_size: int
    hidden_size: int
    name: str = "model.embed_tokens.weight"
    kind: str = "embedding"
    scale: float = 1.0          # the looked-up rows are multiplied by it (in float32)


@dataclass(frozen=True)
class HeadSpec:
    """Output projection; ``tied`` reuses the embedding table
    (src/tokamak/model/transformer.py:154-156)."""

    vocab_size: int
    hidden_size: int
    tied: bool
    name: str = "lm_head.weight"
    kind: str = "linear_head"
    scale: float = 1.0              # the logits are multiplied by it
    softcap: float | None = None    # and then bounded: cap * tanh(logits / cap)


@dataclass(frozen=True)
class BigramEmbeddingSpec:
    """A token table and a table of ``buckets + 1`` rows by hashed pairs: a token's row is ``scale * table[id]`` plus
    the pair row ``(previous id * mul_prev + id * mul_cur) mod buckets``, or the last pair row for a request's first
    token."""

    vocab_size: int
    hidden_size: int
    buckets: int
    mul_prev: int
    mul_cur: int
    name: str = "embed"
    pair_name: str = "bigram"
    scale: float = 1.0
    kind: str = "embedding_bigram"


@EMBEDDINGS.register("embedding")
class Embedding:
    """Row lookup (src/tokamak/model/transformer.py:140), times the spec's ``scale`` where a
    design has one; the rows are widened into the float32 residual stream."""

    GRAPH_SAFE = True

    def weight_bytes(self) -> int:
        return 0          # read by row: a step touches one row per token

    def __init__(self, spec: EmbeddingSpec, tensors: dict[str, torch.Tensor], rt: Runtime):
        self.spec = spec
        self.weight = tensors[spec.name]

    @staticmethod
    def expected_tensors(spec: EmbeddingSpec) -> dict[str, TensorReq]:
        return {spec.name: TensorReq((spec.vocab_size, spec.hidden_size))}

    def forward(self, step) -> torch.Tensor:
        resid = torch.empty((step.n_tokens, self.spec.hidden_size), dtype=torch.float32,
                            device=self.weight.device)
        ops.embed_gather(self.weight, step.token_ids, resid, step.err, scale=self.spec.scale)
        return resid


@EMBEDDINGS.register("embedding_bigram")
class BigramEmbedding:
    """Two row lookups added in float32.  A request's last token is part of its state (one int32 record a slot):
    the next step's first token of the request forms its pair with it."""

    GRAPH_SAFE = True
    TAKES_KEEP = True

    def weight_bytes(self) -> int:
        return 0          # read by row

    def __init__(self, spec: BigramEmbeddingSpec, tensors: dict[str, torch.Tensor], rt: Runtime):
        self.spec = spec
        self.weight = tensors[spec.name]
        self.pairs = tensors[spec.pair_name]

    @staticmethod
    def expected_tensors(spec: BigramEmbeddingSpec) -> dict[str, TensorReq]:
        return {spec.name: TensorReq((spec.vocab_size, spec.hidden_size)),
                spec.pair_name: TensorReq((spec.buckets + 1, spec.hidden_size))}

    def cache_need(self) -> StateNeed:
        return StateNeed((1,), "int32")

    def forward(self, step, cache_view, keep: torch.Tensor | None = None) -> torch.Tensor:
        s = self.spec
        resid = torch.empty((step.n_tokens, s.hidden_size), dtype=torch.float32, device=self.weight.device)
        ops.embed_bigram(self.weight, self.pairs, cache_view.records, step, resid, mul_prev=s.mul_prev, mul_cur=s.mul_cur,
                         scale=s.scale, keep=keep)
        return resid


@HEADS.register("linear_head")
class Head:
    """Logits in float32 for the rows that were asked for
    (src/tokamak/model/transformer.py:173-176).  In bfloat16 the product keeps its
    32-bit accumulators rather than rounding them to bfloat16 first."""

    GRAPH_SAFE = True
    TAKES_OWED_NORM = True     # the product pays an owed norm scale in its epilogue

    def weight_bytes(self) -> int:
        return tensor_bytes(self.weight)

    def __init__(self, spec: HeadSpec, embedding, tensors: dict[str, torch.Tensor], rt: Runtime):
        self.spec = spec
        self.weight = embedding.weight if spec.tied else tensors[spec.name]

    @staticmethod
    def expected_tensors(spec: HeadSpec) -> dict[str, TensorReq]:
        # a tied checkpoint may still carry the head; it is then ignored
        return {spec.name: TensorReq((spec.vocab_size, spec.hidden_size), optional=spec.tied)}

    def forward(self, h: torch.Tensor, step=None) -> torch.Tensor:
        # queued with the products before it; the model flushes the queue before it returns the logits
        logits = linear(h, self.weight, out_dtype=torch.float32, err=getattr(step, "err", None), chain=chain_of(step),
                        queue_plain=True)
        logits = sum_parts(logits, torch.float32)
        if self.spec.scale != 1.0 or self.spec.softcap is not None:
            if not logits.is_contiguous():
                logits = logits.contiguous()
            ops.logits_scale_cap(logits, self.spec.scale, self.spec.softcap)
        return logits
