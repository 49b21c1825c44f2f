"""The gated delta rule: a mixer whose memory is a matrix-valued state per request and head that
every token decays and then corrects towards its own value."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ..cache.manager import StateNeed
from ..csrc import ops
from .base import MIXERS, SWAPPED_GEMM_MAX_TOKENS, Runtime, TensorReq, linear, tensor_bytes


@dataclass(frozen=True)
class GatedDeltaSpec:
    """Sizes, constants and tensor names of one gated-delta-rule mixer.

    ``num_heads`` value heads of ``value_dim`` read ``num_kv_heads`` query/key heads of ``key_dim``
    (value head ``i`` reads q/k head ``i // (num_heads / num_kv_heads)``).  ``conv_taps`` is the
    length of the causal convolution that q, k and v pass; ``unit_eps`` the eps under the root when q
    and k heads are scaled to unit length; ``norm_eps`` the eps of the output norm.

    ``decay_rank``: a decay per head and key channel from a low-rank projection ``W_2 (W_1 h)`` of that rank
    (``decay_names``: the two matrices) instead of one per head; ``dt_bias`` is then ``[heads * key_dim]``.
    ``gate_rank``: the output gate comes from such a projection too (``gate_names``).  ``gate``: its activation,
    ``silu`` or ``sigmoid``.
    """

    hidden_size: int
    num_heads: int
    num_kv_heads: int
    key_dim: int
    value_dim: int
    conv_taps: int
    norm_eps: float
    unit_eps: float = 1e-6
    q_name: str = "q"
    k_name: str = "k"
    v_name: str = "v"
    conv_suffix: str = ".conv"
    beta_name: str = "b"
    decay_name: str = "a"
    decay_log_name: str = "A_log"
    decay_bias_name: str = "dt_bias"
    gate_name: str = "g"
    norm_name: str = "norm"
    o_name: str = "o"
    decay_rank: int | None = None
    decay_names: tuple = ("a1", "a2")
    gate_rank: int | None = None
    gate_names: tuple = ("g1", "g2")
    gate: str = "silu"
    kind: str = "gated_delta"


@MIXERS.register("gated_delta")
class GatedDeltaRule:
    """Per head, with ``S`` the ``[key_dim, value_dim]`` state: ``S <- g S``, ``u = beta (v - S^T k)``,
    ``S <- S + k u^T``, ``o = S^T q`` (the read-out sees the token's own write).  q, k and v pass a
    short causal convolution and silu; q and k heads are scaled to unit length (q also by
    ``key_dim ** -0.5``); ``beta = sigmoid(W_b h)`` and ``g = exp(-exp(A_log) softplus(W_a h + dt_bias))``
    are one number per head (or ``g`` one per head and key channel, then it scales the rows of ``S``).  Every head's ``o``
    is RMS-normed over ``value_dim`` (one weight vector for all heads), multiplied by ``silu(W_g h)`` (or a sigmoid),
    and projected out.

    The request's record in the cache (:class:`~tokamak_b200.cache.manager.StateNeed`, float32, cleared
    when the slot is handed out) holds the state of every head and the last ``conv_taps - 1`` inputs of
    the convolution.  The input projections (of low-rank ones the first halves) are one stacked operand; the second
    halves are one kernel in steps of few tokens and in float32, library products otherwise; convolution, unit norm, beta,
    the decay, the recurrence and the output norm are float32 in every dtype (``csrc/delta.cu``; the
    output stage is the kernel that gated linear attention uses).  :meth:`branch` gives the rows in front of the
    output projection (see :class:`~tokamak_b200.parts.parallel.ParallelMixer`).
    """

    GRAPH_SAFE = True

    def __init__(self, spec: GatedDeltaSpec, prefix: str, tensors: dict[str, torch.Tensor], rt: Runtime):
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"{spec.num_heads} value heads are not a multiple of {spec.num_kv_heads} key heads")
        if spec.key_dim > 256:
            raise ValueError(f"key_dim {spec.key_dim} is beyond the recurrence kernel's limit of 256")
        if not 1 <= spec.conv_taps <= 8:
            raise ValueError(f"a convolution of {spec.conv_taps} taps is not taken (1 to 8)")
        self.spec = spec
        self.rt = rt
        if spec.gate not in ops.GATES:
            raise ValueError(f"unknown gate {spec.gate!r}; known: {', '.join(ops.GATES)}")
        for what, rank in (("decay", spec.decay_rank), ("gate", spec.gate_rank)):
            if rank is not None and not 1 <= rank <= ops.LOW_RANK_MAX:
                raise ValueError(f"a {what} projection of rank {rank} is not taken (1 to {ops.LOW_RANK_MAX})")
        hk, hv, hh = spec.num_kv_heads * spec.key_dim, spec.num_heads * spec.value_dim, spec.num_heads
        t = lambda name: tensors[prefix + name]
        pad = lambda m, dim: torch.nn.functional.pad(m, (0, -m.shape[1] % 8) if dim == 1 else (0, 0, 0, -m.shape[0] % 8))
        # ranks are filled up with zeros to whole eights, and so are the rows of the operand
        mats = [("q", t(spec.q_name)), ("k", t(spec.k_name)), ("v", t(spec.v_name))]
        self.w_decay = self.w_gate = None
        if spec.decay_rank is not None:
            mats.append(("a", pad(t(spec.decay_names[0]), 0)))
            self.w_decay = pad(t(spec.decay_names[1]), 1).contiguous()
        if spec.gate_rank is not None:
            mats.append(("g", pad(t(spec.gate_names[0]), 0)))
            self.w_gate = pad(t(spec.gate_names[1]), 1).contiguous()
        else:
            mats.append(("g", t(spec.gate_name)))
        mats.append(("b", t(spec.beta_name)))
        if spec.decay_rank is None:
            mats.append(("a", t(spec.decay_name)))
        self.offset, at = {}, 0
        for name, m in mats:
            self.offset[name] = at
            at += m.shape[0]
        self.w_in = pad(torch.cat([m for _, m in mats], dim=0), 0).contiguous()
        self.out_width = hv
        self.taps = torch.cat([t(name + spec.conv_suffix).float() for name in (spec.q_name, spec.k_name, spec.v_name)],
                              dim=0).contiguous()
        self.a_log = t(spec.decay_log_name).float().contiguous()
        self.dt_bias = t(spec.decay_bias_name).float().contiguous()
        self.norm_w = t(spec.norm_name)
        self.w_o = t(spec.o_name)
        self.record_floats, _ = ops.delta_record_floats(spec.num_heads, spec.num_kv_heads, spec.key_dim,
                                                        spec.value_dim, spec.conv_taps)

    @staticmethod
    def expected_tensors(spec: GatedDeltaSpec, prefix: str) -> dict[str, TensorReq]:
        w = spec.hidden_size
        hk, hv, hh = spec.num_kv_heads * spec.key_dim, spec.num_heads * spec.value_dim, spec.num_heads
        conv = lambda name: prefix + name + spec.conv_suffix
        out = {
            prefix + spec.q_name: TensorReq((hk, w)),
            conv(spec.q_name): TensorReq((hk, spec.conv_taps), role="bias"),
            prefix + spec.k_name: TensorReq((hk, w)),
            conv(spec.k_name): TensorReq((hk, spec.conv_taps), role="bias"),
            prefix + spec.v_name: TensorReq((hv, w)),
            conv(spec.v_name): TensorReq((hv, spec.conv_taps), role="bias"),
            prefix + spec.beta_name: TensorReq((hh, w)),
            prefix + spec.decay_log_name: TensorReq((hh,), role="bias"),
            prefix + spec.norm_name: TensorReq((spec.value_dim,), role="vector"),
        }
        per_head = hh if spec.decay_rank is None else hh * spec.key_dim
        if spec.decay_rank is None:
            out[prefix + spec.decay_name] = TensorReq((per_head, w))
        else:
            out[prefix + spec.decay_names[0]] = TensorReq((spec.decay_rank, w))
            out[prefix + spec.decay_names[1]] = TensorReq((per_head, spec.decay_rank))
        out[prefix + spec.decay_bias_name] = TensorReq((per_head,), role="bias")
        if spec.gate_rank is None:
            out[prefix + spec.gate_name] = TensorReq((hv, w))
        else:
            out[prefix + spec.gate_names[0]] = TensorReq((spec.gate_rank, w))
            out[prefix + spec.gate_names[1]] = TensorReq((hv, spec.gate_rank))
        out[prefix + spec.o_name] = TensorReq((w, hv))
        return out

    def cache_need(self) -> StateNeed:
        return StateNeed((self.record_floats,), "float32")

    def weight_bytes(self) -> int:
        return tensor_bytes(self.w_in, self.w_decay, self.w_gate, self.taps, self.a_log, self.dt_bias, self.norm_w, self.w_o)

    TAKES_PROJ = True      # the stacked input projection may be part of a wider product (see ParallelMixer)

    def _second_halves(self, proj, at: int) -> tuple:
        """The channel decays' and the gate's low-rank products (``None`` for what is not low-rank)."""
        ws = [("a", self.w_decay), ("g", self.w_gate)]
        factors = [(at + self.offset[name], w) for name, w in ws if w is not None]
        if not factors:
            return None, None
        if proj.dim() == 3 or self.rt.is_f32 or proj.shape[0] <= SWAPPED_GEMM_MAX_TOKENS:
            outs = [o.unsqueeze(0) for o in ops.low_rank(proj, self.rt.dtype, factors)]
        else:
            ops.flush_chains()
            outs = [torch.mm(proj[:, off:off + w.shape[1]], w.t()) for off, w in factors]
        return tuple(outs.pop(0) if w is not None else None for _, w in ws)

    def branch(self, h, step, cache_view, out: torch.Tensor | None = None, out_scale: float = 1.0, proj=None,
               proj_off: int = 0) -> torch.Tensor:
        """The rows in front of the output projection, times ``out_scale``, into ``out`` or a new tensor.  ``proj``:
        a product of ``h`` that holds this part's input projection in its columns from ``proj_off`` on."""
        spec = self.spec
        if proj is None:
            proj, proj_off = linear(h, self.w_in, err=step.err), 0
        off = {name: proj_off + at for name, at in self.offset.items()}
        channel_a, gate = self._second_halves(proj, proj_off)
        q, k, v, beta, g = ops.delta_prepare(
            proj, self.taps, self.a_log, self.dt_bias, cache_view.records, step.tok_req, step.req_q_start,
            step.req_q_len, step.req_slot, step.err, dtype=self.rt.dtype, q_off=off["q"], k_off=off["k"],
            v_off=off["v"], b_off=off["b"], a_off=off["a"], heads=spec.num_heads, kv_heads=spec.num_kv_heads,
            key_dim=spec.key_dim, value_dim=spec.value_dim, unit_eps=spec.unit_eps, q_scale=spec.key_dim ** -0.5,
            channel_a=channel_a)
        o = ops.delta_scan(q, k, v, beta, g, cache_view.records, step.req_q_start, step.req_q_len, step.req_slot,
                           step.err)
        gate_rows, gate_off = (proj, off["g"]) if gate is None else (gate, 0)
        return ops.gla_out(o, gate_rows, gate_off, self.norm_w, spec.norm_eps, self.rt.dtype, out=out,
                           out_scale=out_scale, gate=spec.gate)

    def forward(self, h, step, cache_view):
        return linear(self.branch(h, step, cache_view), self.w_o, err=step.err)
