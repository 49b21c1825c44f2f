"""Two mixers side by side that read the same input; their outputs are added with a factor each."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .base import MIXERS, NormedBranch, NormedSum, Runtime, TensorReq, graph_safe, linear, tensor_bytes, weight_bytes


@dataclass(frozen=True)
class ParallelMixerSpec:
    """``left`` and ``right`` are mixer specs; their tensors lie under ``left_prefix`` / ``right_prefix`` behind the
    part's own prefix; the result is ``left_scale * left(h) + right_scale * right(h)``.  With ``out_norm_eps`` each
    half's output first passes an RMS norm over the model's width with a weight of its own (``out_norm_name`` under
    the half's prefix)."""

    left: object
    right: object
    left_scale: float
    right_scale: float
    left_prefix: str = "left."
    right_prefix: str = "right."
    out_norm_eps: float | None = None
    out_norm_name: str = "out"
    kind: str = "parallel"


@MIXERS.register("parallel")
class ParallelMixer:
    """Both halves must offer ``branch(h, step, cache_view, out, out_scale)`` (the rows in front of their
    output projection, times a factor, written into a column range of a buffer), ``out_width`` and ``w_o``:
    the two output projections are stacked along their inputs once, so that

        ``left_scale * W_l y_l + right_scale * W_r y_r = [W_l | W_r] [left_scale y_l ; right_scale y_r]``

    is one product.  The factors are applied in float32 before the rows are rounded to the engine's dtype.
    The cache need is the dictionary of the halves' needs.

    Halves that declare ``TAKES_PROJ = True`` keep their stacked input projection in ``w_in`` and take
    ``branch(..., proj=, proj_off=)``: the two input projections are then stacked too and run as one product of
    the shared input, each half reading its columns of the result from ``proj_off`` on.

    With output norms there are two output products, and both outputs are left as a
    :class:`~tokamak_b200.parts.base.NormedSum` (the factors are part of the norms' weights): the norm that reads the
    stream next does both norms, the sum and its own normalisation in one kernel.  The block in front of such a norm
    must be one whose norms know it (``pre_norm`` with an RMS norm).
    """

    def __init__(self, spec: ParallelMixerSpec, prefix: str, tensors: dict[str, torch.Tensor], rt: Runtime):
        self.spec = spec
        self.rt = rt
        self.left = MIXERS.get(spec.left.kind)(spec.left, prefix + spec.left_prefix, tensors, rt)
        self.right = MIXERS.get(spec.right.kind)(spec.right, prefix + spec.right_prefix, tensors, rt)
        for half in (self.left, self.right):
            if not (hasattr(half, "branch") and hasattr(half, "out_width") and hasattr(half, "w_o")):
                raise ValueError(f"a {type(half).__name__} cannot be half of a parallel mixer: it has no branch()")
        self.out_norms = None
        if spec.out_norm_eps is None:
            self.w_o = torch.cat([self.left.w_o, self.right.w_o], dim=1).contiguous()
        else:
            self.out_norms = [(scale * tensors[prefix + half + spec.out_norm_name].float()).contiguous()
                              for half, scale in ((spec.left_prefix, spec.left_scale), (spec.right_prefix, spec.right_scale))]
        self.w_in = None
        if all(getattr(half, "TAKES_PROJ", False) for half in (self.left, self.right)):
            n_left = self.left.w_in.shape[0]
            self.w_in = torch.cat([self.left.w_in, self.right.w_in], dim=0).contiguous()
            self.left.w_in, self.right.w_in = self.w_in[:n_left], self.w_in[n_left:]      # one copy in memory
        self.prefill_heads = getattr(self.left, "prefill_heads", None) or getattr(self.right, "prefill_heads", None)

    @staticmethod
    def expected_tensors(spec: ParallelMixerSpec, prefix: str) -> dict[str, TensorReq]:
        out = dict(MIXERS.get(spec.left.kind).expected_tensors(spec.left, prefix + spec.left_prefix))
        out.update(MIXERS.get(spec.right.kind).expected_tensors(spec.right, prefix + spec.right_prefix))
        if spec.out_norm_eps is not None:
            for half in (spec.left_prefix, spec.right_prefix):
                out[prefix + half + spec.out_norm_name] = TensorReq((spec.left.hidden_size,), role="vector")
        return out

    def cache_need(self) -> dict:
        return {"left": self.left.cache_need(), "right": self.right.cache_need()}

    def GRAPH_SAFE(self) -> bool:
        return graph_safe(self.left, self.right)

    def weight_bytes(self) -> int:
        return weight_bytes(self.left, self.right) + tensor_bytes(*(self.out_norms or ()))

    def forward(self, h, step, cache_view):
        if self.out_norms is not None:
            return self._normed(h, step, cache_view)
        n, wl, wr = h.shape[0], self.left.out_width, self.right.out_width
        y = torch.empty((n, wl + wr), dtype=h.dtype, device=h.device)
        if self.w_in is not None:
            proj = linear(h, self.w_in, err=step.err)
            self.left.branch(h, step, cache_view["left"], out=y[:, :wl], out_scale=self.spec.left_scale, proj=proj)
            self.right.branch(h, step, cache_view["right"], out=y[:, wl:], out_scale=self.spec.right_scale, proj=proj,
                              proj_off=self.left.w_in.shape[0])
        else:
            self.left.branch(h, step, cache_view["left"], out=y[:, :wl], out_scale=self.spec.left_scale)
            self.right.branch(h, step, cache_view["right"], out=y[:, wl:], out_scale=self.spec.right_scale)
        return linear(y, self.w_o, err=step.err)

    def _normed(self, h, step, cache_view) -> NormedSum:
        spec = self.spec
        kw = [{}, {}]
        if self.w_in is not None:
            proj = linear(h, self.w_in, err=step.err)
            kw = [dict(proj=proj), dict(proj=proj, proj_off=self.left.w_in.shape[0])]
        y_left = self.left.branch(h, step, cache_view["left"], **kw[0])
        y_right = self.right.branch(h, step, cache_view["right"], **kw[1])
        return NormedSum(NormedBranch(linear(y_left, self.left.w_o, err=step.err), self.out_norms[0], spec.out_norm_eps),
                         NormedBranch(linear(y_right, self.right.w_o, err=step.err), self.out_norms[1], spec.out_norm_eps))
