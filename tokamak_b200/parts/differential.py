"""Differential attention: two attention maps per head over the same values, the second subtracted from the first."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ..cache.manager import KVPagesNeed
from ..csrc import ops
from .attention import paged_attention
from .base import MIXERS, POSITIONS, Runtime, TensorReq, chain_of, graph_safe, linear, tensor_bytes


@dataclass(frozen=True)
class DifferentialAttentionSpec:
    """Sizes and constants of one differential attention mixer.

    Query and key projections hold two pieces of ``head_dim`` elements per head, one per map, head by head; the
    values have ``v_head_dim``.  ``diff`` is what the second map weighs at the start of training and what the heads
    are scaled down by; ``norm_eps`` the eps of the heads' root mean square.  The ``*_name`` fields are the
    tensors' names after the part's prefix."""

    hidden_size: int
    num_heads: int
    num_kv_heads: int
    head_dim: int
    v_head_dim: int
    softmax_scale: float
    position: object
    diff: float
    norm_eps: float
    window: int | None = None
    q_name: str = "q"
    k_name: str = "k"
    v_name: str = "v"
    o_name: str = "o"
    lambda_names: tuple = ("lq1", "lk1", "lq2", "lk2")
    kind: str = "attention_differential"


@MIXERS.register("attention_differential")
class DifferentialAttention:
    """``o = a_1 - lambda a_2`` with ``a_i = softmax(scale q_i k_i^T) v`` and ``lambda = exp(lq1 . lk1) - exp(lq2 . lk2) +
    diff``, every head divided by its root mean square over the value channels, times ``1 - diff``.  Query head ``h``
    reads key/value head ``h // (Hq / Hkv)``.

    One key row of the cache holds both maps' keys, ``[k_1 | k_2]``, and every head has two query rows, ``[q_1 | 0]``
    and ``[0 | q_2]``: the maps are query heads ``2h`` and ``2h + 1`` of an ordinary grouped-query attention, whose
    kernels read every key and value once for both.  In bfloat16 the rows get a size that the tiled kernels take.
    Rotation, layout and page write are one kernel (``csrc/qkv_heads.cu``); difference, norm and scaling another
    (``csrc/map_difference.cu``)."""

    def __init__(self, spec: DifferentialAttentionSpec, prefix: str, tensors: dict[str, torch.Tensor], rt: Runtime):
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"{spec.num_heads} query heads are not a multiple of {spec.num_kv_heads} key/value heads")
        if max(spec.head_dim, spec.v_head_dim) > 512:
            raise ValueError(f"head sizes {spec.head_dim} / {spec.v_head_dim} are beyond the kernels' 512")
        self.spec = spec
        self.rt = rt
        t = lambda name: tensors[prefix + name]
        self.w_in = torch.cat([t(spec.q_name), t(spec.k_name), t(spec.v_name)], dim=0).contiguous()
        self.k_off = 2 * spec.num_heads * spec.head_dim
        self.v_off = self.k_off + 2 * spec.num_kv_heads * spec.head_dim
        self.w_o = t(spec.o_name)
        lq1, lk1, lq2, lk2 = (t(name).double() for name in spec.lambda_names)
        self.map_weight = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + spec.diff)
        self.k_row, self.v_row = 2 * spec.head_dim, spec.v_head_dim
        row = ops.attention_row(max(self.k_row, self.v_row), rt.dtype)
        if rt.dtype == torch.bfloat16 and row in ops.ATTENTION_ROWS:
            self.k_row = self.v_row = row
        self.position = POSITIONS.get(spec.position.kind)(spec.position, tensors, rt)
        if not hasattr(self.position, "rotary_table"):
            raise ValueError(f"position encoding {spec.position.kind!r} does not rotate queries and keys")
        self.halves = getattr(self.position, "PAIRING", "halves") == "halves"
        self.prefill_heads = 2 * spec.num_heads

    @staticmethod
    def expected_tensors(spec: DifferentialAttentionSpec, prefix: str) -> dict[str, TensorReq]:
        h, d, dv = spec.hidden_size, spec.head_dim, spec.v_head_dim
        out = {
            prefix + spec.q_name: TensorReq((2 * spec.num_heads * d, h)),
            prefix + spec.k_name: TensorReq((2 * spec.num_kv_heads * d, h)),
            prefix + spec.v_name: TensorReq((spec.num_kv_heads * dv, h)),
            prefix + spec.o_name: TensorReq((h, spec.num_heads * dv)),
        }
        for name in spec.lambda_names:
            out[prefix + name] = TensorReq((d,), role="bias")
        out.update(POSITIONS.get(spec.position.kind).expected_tensors(spec.position))
        return out

    def cache_need(self) -> KVPagesNeed:
        return KVPagesNeed(self.spec.num_kv_heads, self.k_row, self.spec.window,
                           None if self.v_row == self.k_row else self.v_row)

    def GRAPH_SAFE(self) -> bool:
        return graph_safe(self.position)

    def weight_bytes(self) -> int:
        return tensor_bytes(self.w_in, self.w_o)

    TAKES_OWED_NORM = True     # the input product pays an owed norm scale in its epilogue
    TAKES_THEN_NORM = True     # the output product can add itself to the residual stream

    def forward(self, h, step, cache_view, then_norm=None):
        spec = self.spec
        n, hq = h.shape[0], 2 * spec.num_heads
        proj = linear(h, self.w_in, err=step.err)
        q = torch.empty((n, hq, self.k_row), dtype=self.rt.dtype, device=h.device)
        table, rotary_dim = self.position.rotary_table(step)
        ops.qkv_heads(proj, q, cache_view.k, cache_view.v, step, cache_view.table, q_off=0, k_off=self.k_off,
                      v_off=self.v_off, table=table, rotary_dim=rotary_dim, halves=self.halves, maps=2,
                      k_dim=spec.head_dim, v_dim=spec.v_head_dim)
        att = torch.empty((n, hq, self.v_row), dtype=self.rt.dtype, device=h.device)
        paged_attention(q, att, cache_view, step, scale=spec.softmax_scale, window=spec.window)
        y = ops.map_difference(att, spec.v_head_dim, self.map_weight, spec.norm_eps, 1.0 - spec.diff)
        return linear(y, self.w_o, err=step.err, then_norm=then_norm, chain=chain_of(step))
