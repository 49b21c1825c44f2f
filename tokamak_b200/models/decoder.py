"""A decoder described as data: parts, blocks, and the order in which they run."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ..parts import embedding as _builtin_embedding   # registers the built-in embedding and head
from ..parts.base import (BLOCKS, EMBEDDINGS, HEADS, NORMS, POSITIONS, OwedNorm, Runtime, SumBranch, TensorReq,
                          graph_safe, weight_bytes)


EMBEDDING_CACHE = "embedding"       # the cache key of an embedding that keeps something between steps


@dataclass(frozen=True)
class StreamInput:
    """What joins the residual stream right before a call of the schedule, beside what the block before it left:
    the embedded rows once more (``embedding``, as they were before the first block) and row ``row`` of the float32
    vectors ``[rows, width]`` named ``table`` (one of the model's ``stream_tables``), the same for every token."""

    embedding: bool = False
    table: str | None = None
    row: int = 0


@dataclass(frozen=True)
class LayerCall:
    """One entry of the schedule: which block runs and which cache it uses.

    Naming a block twice runs its weights twice; two calls that name the same
    ``cache`` share keys and values (the later one must be built without key and
    value projections of its own).  ``cache`` is ``None`` for a block that keeps
    nothing between steps.  ``joins`` says what else joins the stream before the block reads it.
    """

    block: str
    cache: str | None
    joins: StreamInput | None = None


@dataclass(frozen=True)
class ModelSpec:
    """A model as data.  Every field but the schedule is a spec with a ``kind`` that one of the
    registries of ``parts/base.py`` resolves; ``embedding_position`` is the seat of a position
    encoding that is added to the embedded rows (``None``: the mixers carry the positions).
    ``streams > 1``: the residual stream is kept in that many float32 copies ``[streams, tokens, width]``, all
    equal to the embedded rows at the start; the blocks and the last norm must know such a stream (the
    ``hyper`` block, the ``layernorm`` norm, which reads the sum of the copies at the end).  ``stream_tables``:
    ``(tensor name, rows)`` of the vectors that calls of the schedule add to the stream (``StreamInput``)."""

    embedding: object                  # an embedding spec (vocab_size, hidden_size, kind, ...)
    blocks: tuple                      # block specs, each with a unique ``name``
    schedule: tuple                    # LayerCall entries, in execution order
    final_norm: object
    final_norm_name: str
    head: object                       # a head spec (vocab_size, kind, ...)
    embedding_position: object = None
    streams: int = 1
    stream_tables: tuple = ()

    def __post_init__(self) -> None:
        names = [b.name for b in self.blocks]
        if len(set(names)) != len(names):
            raise ValueError("block names must be unique")
        for call in self.schedule:
            if call.block not in names:
                raise ValueError(f"the schedule names an unknown block {call.block!r}")
            if call.cache == EMBEDDING_CACHE:
                raise ValueError(f"the cache key {EMBEDDING_CACHE!r} is the embedding's")
            if call.joins is not None:
                if self.streams > 1:
                    raise ValueError("nothing else joins a stream that is kept in several copies")
                rows = dict(self.stream_tables).get(call.joins.table, 0)
                if call.joins.table is not None and not 0 <= call.joins.row < rows:
                    raise ValueError(f"the model's stream tables have no row {call.joins.row} of {call.joins.table!r}")


def flat_needs(key, need) -> list[tuple]:
    """``(cache key, need)`` pairs of a block's need.  A block that keeps several things per request (pages
    for one mixer, state records for another, records of its own) declares a dictionary ``{name: need}``,
    nested at will; its entries become the cache keys ``key/name``."""
    if isinstance(need, dict):
        return [pair for name, sub in need.items() for pair in flat_needs(f"{key}/{name}", sub)]
    return [] if need is None else [(key, need)]


def views_of(cache, key, need):
    """The view, or the dictionary of views in the shape of the block's need."""
    if isinstance(need, dict):
        return {name: views_of(cache, f"{key}/{name}", sub) for name, sub in need.items()}
    return None if need is None else cache.view(key)


class DecoderModel:
    """Embedding, the scheduled blocks, final norm and head
    (src/tokamak/model/transformer.py:112-176), built from a :class:`ModelSpec`."""

    def __init__(self, spec: ModelSpec, tensors: dict[str, torch.Tensor], rt: Runtime):
        self.spec = spec
        self.rt = rt
        self.embedding = EMBEDDINGS.get(spec.embedding.kind)(spec.embedding, tensors, rt)
        self.embedding_position = None
        if spec.embedding_position is not None:
            pos = spec.embedding_position
            self.embedding_position = POSITIONS.get(pos.kind)(pos, tensors, rt)
            if not hasattr(self.embedding_position, "add_to_embedding"):
                raise ValueError(f"position encoding {pos.kind!r} cannot sit at the embedding: "
                                 f"it has no add_to_embedding")
        self.blocks = {b.name: BLOCKS.get(b.kind)(b, tensors, rt) for b in spec.blocks}
        self.final_norm = NORMS.get(spec.final_norm.kind)(spec.final_norm, spec.final_norm_name,
                                                          tensors, rt)
        self.head = HEADS.get(spec.head.kind)(spec.head, self.embedding, tensors, rt)
        self._needs = {name: block.cache_need() for name, block in self.blocks.items()}
        self._embedding_need = self.embedding.cache_need() if hasattr(self.embedding, "cache_need") else None
        self.stream_tables = {name: tensors[name].float().contiguous() for name, _ in spec.stream_tables}
        self._keeps_embedding = any(call.joins is not None and call.joins.embedding for call in spec.schedule)

    @staticmethod
    def expected_tensors(spec: ModelSpec) -> dict[str, TensorReq]:
        out: dict[str, TensorReq] = {}
        out.update(EMBEDDINGS.get(spec.embedding.kind).expected_tensors(spec.embedding))
        if spec.embedding_position is not None:
            pos = spec.embedding_position
            out.update(POSITIONS.get(pos.kind).expected_tensors(pos))
        for b in spec.blocks:
            out.update(BLOCKS.get(b.kind).expected_tensors(b))
        out.update(NORMS.get(spec.final_norm.kind).expected_tensors(spec.final_norm,
                                                                    spec.final_norm_name))
        for name, rows in spec.stream_tables:
            out[name] = TensorReq((rows, spec.embedding.hidden_size), role="bias")
        out.update(HEADS.get(spec.head.kind).expected_tensors(spec.head))
        return out

    def parts(self) -> list:
        """Every part a step runs, a block once per call of the schedule."""
        out = [self.embedding] + ([self.embedding_position] if self.embedding_position is not None else [])
        out += [self.blocks[call.block] for call in self.spec.schedule]
        return out + [self.final_norm, self.head]

    def graph_safe(self) -> bool:
        """Whether a step of single next tokens may be replayed from a CUDA graph: every part
        has to declare it (``GRAPH_SAFE`` in ``parts/base.py``)."""
        return graph_safe(*self.parts())

    def step_weight_bytes(self) -> int:
        """Bytes of weights that one step reads in full: every scheduled call's, the final norm's
        and the head's (what the parts report through ``weight_bytes``)."""
        return weight_bytes(*self.parts())

    def cache_needs(self) -> dict[str, object]:
        """Cache key -> need, checked for agreement between calls that share a key."""
        needs: dict[str, object] = dict(flat_needs(EMBEDDING_CACHE, self._embedding_need))
        for call in self.spec.schedule:
            need = self.blocks[call.block].cache_need()
            if need is None:
                if call.cache is not None:
                    raise ValueError(f"block {call.block!r} keeps no cache but is given {call.cache!r}")
                continue
            if call.cache is None:
                raise ValueError(f"block {call.block!r} needs a cache and the schedule names none")
            for key, sub in flat_needs(call.cache, need):
                if key in needs and needs[key] != sub:
                    raise ValueError(f"cache {key!r} is shared by blocks with different needs")
                needs.setdefault(key, sub)
        return needs

    def _embed(self, step) -> tuple[torch.Tensor, torch.Tensor | None]:
        """The embedded rows and, where a call of the schedule adds them once more, a copy of them."""
        kw, keep = {}, None
        if self._embedding_need is not None:
            kw["cache_view"] = views_of(step.cache, EMBEDDING_CACHE, self._embedding_need)
        if self._keeps_embedding and self.embedding_position is None and getattr(self.embedding, "TAKES_KEEP", False):
            keep = kw["keep"] = torch.empty((step.n_tokens, self.spec.embedding.hidden_size), dtype=torch.float32,
                                            device=self.rt.device)
        resid = self.embedding.forward(step, **kw)
        if self.embedding_position is not None:
            self.embedding_position.add_to_embedding(resid, step)
        if self._keeps_embedding and keep is None:
            keep = resid.clone()
        return resid, keep

    def _join(self, resid, pending, joins: StreamInput | None, embedded, norm):
        """What ``norm`` finds pending: the branch that is waiting together with what ``joins`` names.  A norm that
        adds it all in its own kernel gets a :class:`SumBranch`; in front of any other the rest is added here."""
        if joins is not None:
            extra = embedded if joins.embedding else None
            vector = self.stream_tables[joins.table][joins.row] if joins.table is not None else None
            if pending is None or isinstance(pending, (torch.Tensor, SumBranch)):
                terms = pending.terms if isinstance(pending, SumBranch) else (() if pending is None else (pending,))
                pending = SumBranch(terms, extra, vector)
            else:
                SumBranch((), extra, vector).settle(resid)      # the branch joins later; the sum is the same
        if isinstance(pending, SumBranch) and not getattr(norm, "TAKES_SUM", False):
            pending.settle(resid)
            pending = None
        return pending

    def forward(self, step) -> torch.Tensor:
        """Float32 logits ``[len(step.logits_rows), vocab]`` for the rows asked for."""
        resid, embedded = self._embed(step)
        if self.spec.streams > 1:
            resid = resid.unsqueeze(0).repeat(self.spec.streams, 1, 1)
        pending = None
        schedule = self.spec.schedule
        for i, call in enumerate(schedule):
            view = views_of(step.cache, call.cache, self._needs[call.block]) if call.cache is not None else None
            block = self.blocks[call.block]
            pending = self._join(resid, pending, call.joins, embedded, getattr(block, "entry_norm", None))
            if getattr(block, "TAKES_NEXT_NORM", False):
                # the norm that will consume what the block leaves pending: the next block's, or the last; none
                # where more joins the stream before it or the reader behind it cannot pay an owed scale
                after = self.blocks[schedule[i + 1].block] if i + 1 < len(schedule) else None
                next_norm = getattr(after, "entry_norm", None) if after is not None else self.final_norm
                if after is not None and (schedule[i + 1].joins is not None or not getattr(after, "entry_takes_owed", True)):
                    next_norm = None
                resid, pending = block.forward(resid, pending, step, view, next_norm=next_norm)
            else:
                resid, pending = block.forward(resid, pending, step, view)
        if step.n_want == 0:
            return torch.empty((0, self.spec.head.vocab_size), dtype=torch.float32, device=resid.device)
        pending = self._join(resid, pending, None, None, self.final_norm)
        # every request brings one token and wants it: the wanted rows are all rows, in order
        all_rows = step.n_want == step.n_tokens and step.max_q_len == 1
        h = self.final_norm.add_norm(resid, pending, rows=None if all_rows and isinstance(pending, OwedNorm) else step.logits_rows)
        if isinstance(h, OwedNorm) and not getattr(self.head, "TAKES_OWED_NORM", False):
            h = h.materialize()
        logits = self.head.forward(h, step)
        from ..csrc import ops
        ops.flush_chains()          # products that are still queued: the caller reads the logits
        return logits
