"""The Sofinex design on the GPU: every mechanism's kernels against the plain implementation, then whole
models under every way of cutting and batching their requests, and generation through the engine's entry
point."""

from __future__ import annotations

import functools
import json
import math
import subprocess
import sys
import tempfile
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import sofinex_configs as sc
import traces
from helpers import assert_logits_close, random_tokens
from plain import sofinex_plain as plain

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
_TMP = []


@functools.lru_cache(maxsize=None)
def folder_of(tag: str, dtype: str) -> Path:
    tmp = tempfile.TemporaryDirectory(prefix=f"sx_{tag}_{dtype}_")
    _TMP.append(tmp)
    return Path(sc.write_folder(tmp.name, tag, dtype))


@functools.lru_cache(maxsize=None)
def _truth(folder: str, tokens: tuple):
    """Logits of the whole sequence, and for every position how close any router came to another choice at
    or before it (a choice made otherwise early in a sequence reaches later positions through keys and states)."""
    cfg, w = plain.load_folder(folder)
    margins = []
    logits = plain.forward(cfg, w, list(tokens), margins_out=margins)
    risk = torch.stack(margins).min(0).values.cummin(0).values if margins else torch.full((len(tokens),), math.inf)
    return logits, risk


# bfloat16: a row is judged against what rounding alone costs in its request (the plain implementation
# rounding at every product's input and output): the level is the worst row of the request, the limit four
# times that and never below the level of a well-conditioned row.  A wrong key, state or expert moves a row by about
# its spread.  So does a router that rounding tips elsewhere than in the plain implementation: the few rows
# beyond the limit that have a router within CLOSE of another choice, at or before them, are let through, counted.
BF16_FLOOR_RMS, BF16_FLOOR_MAX, BF16_TIMES = 0.05, 0.2, 4.0
CLOSE, TIPPED_ROWS, TIPPED_SHARE = 0.01, 2, 0.06


@functools.lru_cache(maxsize=None)
def _rounding_level(folder: str, tokens: tuple) -> tuple[float, float]:
    cfg, w = plain.load_folder(folder)
    want = _truth(folder, tokens)[0]
    rounded = plain.forward(cfg, w, list(tokens), ROUND=plain.bf16_round)
    rel = (rounded - want).abs() / want.std(dim=-1, keepdim=True).clamp_min(1e-6)
    return rel.pow(2).mean(-1).sqrt().max().item(), rel.max().item()


def check_rows(results, rows, reqs, folder, dtype, what) -> int:
    n, tipped = 0, []
    for step in sorted(rows):
        got = torch.from_numpy(np.asarray(results[step])).double()
        for i, (rid, p) in enumerate(rows[step]):
            where = f"{what}: step {step}, request {rid!r}, position {p}"
            toks = tuple(int(t) for t in reqs[rid])
            logits, risk = _truth(str(folder), toks)
            want = logits[p]
            n += 1
            if dtype == "float32":
                assert_logits_close(got[i:i + 1], want[None], dtype, where)
                continue
            assert torch.isfinite(got[i]).all(), where
            mine = (got[i] - want).abs() / want.std().clamp_min(1e-6)
            base_rms, base_max = _rounding_level(str(folder), toks)
            rms = mine.pow(2).mean().sqrt().item()
            ok = (rms <= max(BF16_FLOOR_RMS, BF16_TIMES * base_rms)
                  and mine.max().item() <= max(BF16_FLOOR_MAX, BF16_TIMES * base_max))
            if not ok and risk[p].item() < CLOSE:
                tipped.append((rid, p))
                continue
            assert ok, (f"{where}: off by {rms:.3e} (rms) and {mine.max().item():.3e} (max) of the row's spread; "
                        f"rounding alone costs up to {base_rms:.3e} and {base_max:.3e}")
    assert len(tipped) <= max(TIPPED_ROWS, TIPPED_SHARE * n), f"{what}: {len(tipped)} of {n} rows are off: {tipped}"
    return n


def dev(x, dtype=None):
    return x.to("cuda", dtype) if dtype is not None else x.to("cuda")


def i32(v):
    return torch.tensor(list(v), dtype=torch.int32, device="cuda")


def close(got, want, dtype, scale=1.0):
    got, want = got.detach().cpu().double(), want.double()
    tol = (2e-5 if dtype == "float32" else 2e-2) * scale
    err = (got - want).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), f"off by {err:.3e}"


def fake_step(q_lens, slots, starts, heads=1):
    """What a kernel reads of a step: requests of ``q_lens`` tokens in ``slots``, continuing at ``starts``."""
    from tokamak_b200.csrc import ops
    tok_req, pos, q_start = [], [], []
    at = 0
    for r, (n, s) in enumerate(zip(q_lens, starts)):
        q_start.append(at)
        tok_req += [r] * n
        pos += list(range(s, s + n))
        at += n
    kv_len = [s + n for s, n in zip(starts, q_lens)]
    rec, n_parts, n_split = ops.prefill_tc_records(q_start, q_lens, kv_len, slots, heads=heads,
                                                   sms=ops.sm_count(torch.device("cuda", 0)))
    return SimpleNamespace(tok_req=i32(tok_req), positions=i32(pos), req_q_start=i32(q_start), req_q_len=i32(q_lens),
                           req_slot=i32(slots), req_kv_len=i32(kv_len), max_kv_len=max(kv_len),
                           err=torch.zeros(4, dtype=torch.int32, device="cuda"), max_q_len=max(q_lens), n_tokens=at,
                           scratch={}, decode_items=i32([s for s, n in zip(q_start, q_lens) if n == 1]),
                           prefill_items=i32([s + j for s, n in zip(q_start, q_lens) if n > 1 for j in range(n)]),
                           prefill_tc=ops.PrefillItems(torch.from_numpy(rec).cuda(), n_parts, n_split),
                           prefill_tiles=i32([x for r, n in enumerate(q_lens) if n > 1 for t in range(-(-n // 64)) for x in (r, t)]))


def run_in_steps(seqs, slots, cuts, fn, heads=1):
    """Feed sequences (``[T, ...]`` each, one per request) through ``fn(rows of the step, step)`` cut into steps:
    ``cuts[r]`` lists request r's portion sizes, step by step (0: the request sits the step out).  Returns
    the outputs put together again per request."""
    outs = [[] for _ in seqs]
    fed = [0] * len(seqs)
    for s in range(max(len(c) for c in cuts)):
        live = [r for r in range(len(seqs)) if s < len(cuts[r]) and cuts[r][s] > 0]
        step = fake_step([cuts[r][s] for r in live], [slots[r] for r in live], [fed[r] for r in live], heads)
        rows = torch.cat([seqs[r][fed[r]:fed[r] + cuts[r][s]] for r in live])
        y = fn(rows, step)
        assert step.err.tolist()[0] == 0
        at = 0
        for r in live:
            outs[r].append(y[at:at + cuts[r][s]].detach().cpu())
            at += cuts[r][s]
            fed[r] += cuts[r][s]
    assert fed == [len(x) for x in seqs]
    return [torch.cat(o) for o in outs]


def _part(registry, spec, weights, dtype, prefix="m."):
    from tokamak_b200.parts.base import Runtime
    cls = registry.get(spec.kind)
    tensors = {}
    for name, req in cls.expected_tensors(spec, prefix).items():
        t = weights[name[len(prefix):]]
        assert tuple(t.shape) == tuple(req.shape), name
        tensors[name] = dev(t, TORCH[dtype] if req.role == "matrix" else torch.float32)
    return cls(spec, prefix, tensors, Runtime(device=torch.device("cuda"), dtype=TORCH[dtype]))


def _rounded(gen, dtype):
    return lambda *s, std=1.0: (torch.randn(*s, generator=gen) * std).to(TORCH[dtype]).float()


def _doubles(w):
    return {k: t.double() for k, t in w.items()}


# ======================================================================= mechanisms alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,ff", [(3, 48, 72), (1, 128, 256), (40, 128, 384), (70, 54, 50), (600, 256, 11008 // 8), (4500, 64, 1536)])
def test_dense_feed_forward_with_the_exact_gelu(dtype, n, width, ff):
    from tokamak_b200.parts.base import FEED_FORWARDS
    from tokamak_b200.parts.feedforward import MlpSpec
    gen = torch.Generator().manual_seed(n + ff)
    rnd = _rounded(gen, dtype)
    w = {"up": rnd(ff, width, std=1.5 / width ** 0.5), "down": rnd(width, ff, std=1.5 / ff ** 0.5)}
    x = rnd(n, width)
    part = _part(FEED_FORWARDS, MlpSpec(width, ff, activation="gelu"), w, dtype)
    got = part.forward(dev(x, TORCH[dtype]), fake_step([n], [0], [0]))
    got = got.float().sum(0) if got.dim() == 3 else got.float()
    close(got, plain.dense_ff(x.double(), _doubles(w)), dtype)
    from tokamak_b200.csrc import ops
    z = torch.linspace(-6, 6, 1000).repeat(2, 1)
    act = ops.unary_act(dev(z), torch.float32, "gelu").cpu().double()
    assert (act - plain.gelu_exact(z.double())).abs().max() < 1e-6          # the tanh form is off by 4e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,heads,dv,row", [(5, 3, 14, 14), (1, 2, 96, 128), (33, 4, 128, 128), (7, 1, 5, 64), (2, 5, 300, 300)])
def test_difference_of_two_maps(dtype, n, heads, dv, row):
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(dv)
    a = _rounded(gen, dtype)(n, 2 * heads, row)
    got = ops.map_difference(dev(a, TORCH[dtype]), dv, 0.7, 1e-5, 0.6)
    d = a.double()[..., :dv]
    want = plain.unit_rms(d[:, ::2] - 0.7 * d[:, 1::2], 1e-5) * 0.6
    close(got, want.reshape(n, heads * dv), dtype)
    wide = torch.zeros(n, heads * dv + 8, dtype=TORCH[dtype], device="cuda")
    ops.map_difference(dev(a, TORCH[dtype]), dv, 0.7, 1e-5, 0.6, out=wide[:, 4:4 + heads * dv])
    assert torch.equal(wide[:, 4:4 + heads * dv], got) and not wide[:, :4].any() and not wide[:, 4 + heads * dv:].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width", [(5, 48), (3, 54), (300, 256), (2, 4096), (9, 8200)])
def test_two_normed_branches_their_sum_and_the_next_norm(dtype, n, width):
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(width + n)
    rnd = _rounded(gen, dtype)
    x, a, b = torch.randn(n, width, generator=gen), rnd(n, width, std=3.0), rnd(n, width, std=0.2)
    wa, wb, wn = (torch.randn(width, generator=gen) for _ in range(3))
    sum_ = x.double() + plain.unit_rms(a.double(), 1e-5) * wa + plain.unit_rms(b.double(), 1e-5) * wb
    want = plain.unit_rms(sum_, 1e-4) * wn
    parts = lambda t: dev(torch.stack([0.25 * t, 0.5 * t, 0.25 * t]))
    for fa, fb in ((lambda t: dev(t, TORCH[dtype]),) * 2, (parts, lambda t: dev(t, TORCH[dtype])), (parts, parts)):
        resid, out = dev(x), torch.empty(n, width, dtype=TORCH[dtype], device="cuda")
        ops.branch_pair_norm_add(resid, fa(a), dev(wa), fb(b), dev(wb), 1e-5, dev(wn), out, 1e-4)
        close(resid, sum_, "float32")
        close(out, want, dtype)
        pick = sorted({0, n // 2, n - 1})
        resid, some = dev(x), torch.empty(len(pick), width, dtype=TORCH[dtype], device="cuda")
        ops.branch_pair_norm_add(resid, fa(a), dev(wa), fb(b), dev(wb), 1e-5, dev(wn), some, 1e-4, rows=i32(pick))
        assert torch.equal(resid, dev(x)) and torch.equal(some, out[pick])


def _marked(gen, dtype, T, width, marks, queries):
    """Rows whose channels 0 and 2 mark keys and channel 1 marks queries, and a second, unmarked request."""
    rnd = _rounded(gen, dtype)
    seqs = [rnd(T, width, std=0.5), rnd(77, width, std=0.5)]
    for s in seqs:
        s[:, :3] = 0.0
    for channel, at in marks:
        seqs[0][at, channel] = 8.0
    seqs[0][queries, 1] = 8.0
    return seqs


def _edges(keys, window, page, T):
    """Positions around both edges of the window behind every marked key, at page borders, and the last."""
    at = {4 * page - 1, 4 * page, T - 1}
    for k in keys:
        at |= {k + 1, k + window - 2, k + window - 1, k + window, k + window + 1}
    return sorted(p for p in at if max(keys) < p < T)


def _attention_runs(part, seqs, dtype, page, rows, window, heads):
    """The mixer over a cache of its own: whole prompts, portions down to two tokens beside another request, and
    the marked stretch token by token; pages in a random order, stale values in those not yet written."""
    from tokamak_b200.cache.device import KVView
    T, T2 = len(seqs[0]), len(seqs[1])
    gen = torch.Generator().manual_seed(T)
    need = part.cache_need()
    order, pages = torch.randperm(96, generator=gen).int(), -(-T // page)
    table = torch.full((4, 60), -1, dtype=torch.int32)
    table[2, :pages], table[0, :-(-T2 // page)] = order[:pages], order[pages:pages - (-T2 // page)]
    cuts = [[[T], [T2]], [[7, 2, 30, 2, 64, 3, 2, T - 110], [2, 40, 0, 2, 2, T2 - 46]],
            [[16] + [1] * (T - 16), [40, 0, 1, 2] + [1] * (T2 - 43)]]
    width = seqs[0].shape[1]
    for cut in cuts:
        k = torch.full((96, need.n_kv_heads, page, need.head_dim), float("nan"), dtype=TORCH[dtype], device="cuda")
        v = torch.full((96, need.n_kv_heads, page, need.value_dim), float("nan"), dtype=TORCH[dtype], device="cuda")
        view = KVView(k, v, dev(table), page, window)
        yield run_in_steps(seqs, [2, 0], cut, lambda x, step: torch.as_tensor(rows(part, dev(x, TORCH[dtype]), step, view)).float(),
                           heads)


def _sum(y, n):
    return y.float().sum(0) if y.dim() == 3 else y.float()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,window,page,dims,scaling", [
    (3, 1, 10, 14, 9, 4, 6, {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 60}),
    (4, 2, 32, 64, 48, 16, 32, {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 512}),
    (4, 4, 16, 20, 17, 16, 12, None), (6, 2, 64, 128, 64, 32, 64, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}),
    (2, 1, 30, 100, 1, 16, 0, None), (2, 2, 70, 24, 33, 8, 40, None), (16, 2, 24, 40, 300, 16, 24, None)])
def test_differential_attention_with_keys_that_stand_out_at_the_windows_edges(dtype, H, G, d, dv, window, page, dims, scaling):
    """A marked key of its own for either map, and marked queries around the two edges of each one's window: the
    marked pair's score beats every other, so that a key that one map loses or sees too long moves the row by its
    whole spread (which is checked in the oracle)."""
    from tokamak_b200.parts.base import MIXERS
    from tokamak_b200.parts.differential import DifferentialAttentionSpec
    from tokamak_b200.parts.position import NoPositionSpec, RopeHalvesSpec, WaveScaling
    gen = torch.Generator().manual_seed(H * 100 + d)
    rnd = _rounded(gen, dtype)
    width, T, eps, diff, base = 72, 150, 1e-5, 0.4, 1e5
    w = {"q": rnd(2 * H * d, width, std=0.1), "k": rnd(2 * G * d, width, std=0.1), "v": rnd(G * dv, width, std=0.3),
         "o": rnd(width, H * dv, std=0.2)}
    for name in ("lq1", "lk1", "lq2", "lk2"):
        w[name] = 0.4 * torch.randn(d, generator=gen) / d ** 0.25
    w["q"][:, 1], w["k"][:, 0], w["k"][:, 2] = 0.0, 0.0, 0.0
    w["q"][d - 1::d, 1] = 1.0                                # the piece's last element: unrotated, or turned slowest
    for g in range(G):
        w["k"][2 * g * d + d - 1, 0] = 1.0                   # the first map's key
        w["k"][(2 * g + 1) * d + d - 1, 2] = 1.0             # the second map's
    marks = [(0, 19), (2, 24)]
    queries = _edges([19, 24], window, page, T)
    seqs = _marked(gen, dtype, T, width, marks, queries)
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": 0.45, "diff": diff, "mask": {"size": window},
         "rot": {"base": base, "dims": dims, "scaling": scaling}}
    wd = _doubles(w)
    want = [plain.differential_attention(s.double(), wd, m, eps, torch.arange(len(s))) for s in seqs]
    for at, other in [(k + window - 1, window - 1) for k in (19, 24)] + [(k + window, window + 1) for k in (19, 24)]:
        if at in queries and other > 0:          # a window that is one token off would show
            off = plain.differential_attention(seqs[0].double(), wd, {**m, "mask": {"size": other}}, eps, torch.arange(T))
            assert (off[at] - want[0][at]).abs().max() > 0.3 * want[0].std(), (at, other)
    pos = NoPositionSpec() if dims == 0 else RopeHalvesSpec(dims, base, scaling=None if scaling is None else WaveScaling(**scaling))
    part = _part(MIXERS, DifferentialAttentionSpec(hidden_size=width, num_heads=H, num_kv_heads=G, head_dim=d, v_head_dim=dv,
                                                   softmax_scale=0.45, position=pos, diff=diff, norm_eps=eps, window=window), w, dtype)
    assert abs(part.map_weight - float(plain.map_weight(wd, diff))) < 1e-6
    rows = lambda p, x, step, view: _sum(p.forward(x, step, view), x.shape[0])
    for got in _attention_runs(part, seqs, dtype, page, rows, window, 2 * H):
        for g, ref in zip(got, want):
            close(g, ref, dtype, scale=3.0 if dtype == "float32" else 4.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,window,page,dims,scaling", [
    (4, 2, 12, 20, 17, 4, 8, {"factor": 4.0, "original": 40, "fast": 8.0, "slow": 1.0}),
    (4, 1, 64, 64, 45, 16, 64, {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0}),
    (8, 2, 88, 72, 64, 16, 48, {"factor": 16.0, "original": 128, "fast": 32.0, "slow": 1.0}),
    (3, 3, 18, 6, 1, 8, 18, None), (2, 2, 40, 128, 33, 32, 40, None), (2, 1, 140, 24, 300, 16, 0, None)])
def test_attention_with_a_norm_behind_the_rotation_and_sinks(dtype, H, G, d, dv, window, page, dims, scaling):
    """As above, for queries and keys that are divided by their root mean square after a rotation that also changes
    their length, and a sink in the denominator."""
    from tokamak_b200.parts.attention import GatedAttentionSpec
    from tokamak_b200.parts.base import MIXERS
    from tokamak_b200.parts.position import NoPositionSpec, RopeHalvesSpec, YarnScaling
    gen = torch.Generator().manual_seed(H * 100 + d)
    rnd = _rounded(gen, dtype)
    width, T, eps, base, scale = 72, 150, 1e-5, 1e6, 18.0 / d
    w = {"q": rnd(H * d, width, std=0.15), "k": rnd(G * d, width, std=0.15), "v": rnd(G * dv, width, std=0.3),
         "o": rnd(width, H * dv, std=0.2), "sink": 3.0 + 2.0 * torch.randn(H, generator=gen)}
    w["q"][:, 1], w["k"][:, 0] = 0.0, 0.0
    w["q"][d - 1::d, 1] = 4.0
    w["k"][d - 1::d, 0] = 4.0
    queries = _edges([19], window, page, T)
    seqs = _marked(gen, dtype, T, width, [(0, 19)], queries)
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": scale, "mask": {"size": window},
         "rot": {"base": base, "dims": dims, "scaling": scaling}}
    wd = _doubles(w)
    want = [plain.sink_attention(s.double(), wd, m, eps, torch.arange(len(s))) for s in seqs]
    for at, other in ((19 + window - 1, window - 1), (19 + window, window + 1)):
        if at in queries and other > 0:
            off = plain.sink_attention(seqs[0].double(), wd, {**m, "mask": {"size": other}}, eps, torch.arange(T))
            assert (off[at] - want[0][at]).abs().max() > 0.3 * want[0].std(), (at, other)
    no_sink = plain.sink_attention(seqs[0].double(), {**wd, "sink": wd["sink"] - 1e9}, m, eps, torch.arange(T))
    assert (no_sink - want[0]).abs().max() > 0.3 * want[0].std()
    pos = NoPositionSpec() if dims == 0 else RopeHalvesSpec(dims, base, scaling=None if scaling is None else YarnScaling(**scaling))
    part = _part(MIXERS, GatedAttentionSpec(hidden_size=width, num_heads=H, num_kv_heads=G, head_dim=d, v_head_dim=dv,
                                            softmax_scale=scale, position=pos, head_norm_eps=eps, head_norm_weight=False,
                                            norm_after=True, sinks=True, window=window, pad_rows=True), w, dtype)
    rows = lambda p, x, step, view: _sum(p.forward(x, step, view), x.shape[0])
    for got in _attention_runs(part, seqs, dtype, page, rows, window, H):
        for g, ref in zip(got, want):
            close(g, ref, dtype, scale=3.0 if dtype == "float32" else 4.0)


# ======================================================================= the delta rule with channel decays

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,parts,factors", [(3, 2, [(24, 40), (8, 130)]), (1, 1, [(128, 512), (128, 512)]), (70, 0, [(8, 9)]),
                                             (64, 3, [(48, 64), (16, 200)]), (9, 0, [(256, 33), (40, 77)])])
def test_second_halves_of_low_rank_projections(dtype, n, parts, factors):
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(n)
    rnd = _rounded(gen, dtype)
    ranks = [r for r, _ in factors]
    off = [12 + sum(ranks[:i]) for i in range(len(ranks))]
    x = rnd(n, 20 + sum(ranks))
    ws = [rnd(c, r, std=r ** -0.5) for r, c in factors]
    proj = dev(torch.stack([x / parts] * parts)) if parts else dev(x, TORCH[dtype])
    got = ops.low_rank(proj, TORCH[dtype], [(o, dev(w, TORCH[dtype])) for o, w in zip(off, ws)])
    for o, w, g in zip(off, ws, got):
        assert g.dtype == torch.float32
        close(g, x[:, o:o + w.shape[1]].double() @ w.double().T, dtype, scale=0.5 if dtype == "bfloat16" else 1.0)


CUTS = [[5, 1, 1, 0, 2, 7, 1, 40, 2], [1, 1, 3, 9, 0, 2, 0, 3, 30], [16, 1, 0, 0, 1, 1, 2, 9]]    # the second step is single tokens only
SLOTS = [2, 0, 3]


def _delta_weights(gen, dtype, width, H, G, dk, dv, taps, ra, rg):
    rnd = _rounded(gen, dtype)
    s = 1.5 / width ** 0.5
    w = {"q": rnd(G * dk, width, std=s), "k": rnd(G * dk, width, std=s), "v": rnd(H * dv, width, std=s),
         "b": rnd(H, width, std=2 * s), "A_log": 0.5 * torch.randn(H, generator=gen),
         "norm": 1 + 0.3 * torch.randn(dv, generator=gen), "dt_bias": torch.randn(H * dk, generator=gen) - 2.0,
         "a1": rnd(ra, width, std=s), "a2": rnd(H * dk, ra, std=1.5 / ra ** 0.5), "g1": rnd(rg, width, std=s),
         "g2": rnd(H * dv, rg, std=1.5 / rg ** 0.5), "o": rnd(width, H * dv, std=(H * dv) ** -0.5)}
    for n, c in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
        w[n + ".conv"] = 0.6 * torch.randn(c, taps, generator=gen)
    return w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,taps,ra,rg", [(4, 2, 12, 10, 3, 5, 11), (3, 1, 7, 9, 1, 8, 3), (2, 2, 64, 64, 4, 20, 28),
                                                  (4, 4, 130, 33, 2, 16, 40), (2, 1, 256, 20, 6, 7, 8), (8, 4, 128, 128, 4, 128, 128)])
def test_delta_rule_with_a_decay_per_channel(dtype, H, G, dk, dv, taps, ra, rg):
    """The mixer cut into steps beside other requests (down to single tokens, with a step of single tokens only, and
    with pauses), in slots that held another request's state before; and a portion of many tokens."""
    from tokamak_b200.parts.base import MIXERS
    from tokamak_b200.parts.delta import GatedDeltaSpec
    gen = torch.Generator().manual_seed(H * dk + dv)
    width, eps = 96, 1e-5
    w = _delta_weights(gen, dtype, width, H, G, dk, dv, taps, ra, rg)
    part = _part(MIXERS, GatedDeltaSpec(hidden_size=width, num_heads=H, num_kv_heads=G, key_dim=dk, value_dim=dv, conv_taps=taps,
                                        norm_eps=eps, decay_rank=ra, gate_rank=rg, gate="sigmoid"), w, dtype)
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv}
    rnd = _rounded(gen, dtype)
    seqs = [rnd(sum(c), width) for c in CUTS]
    wd = _doubles(w)
    ROUND = plain.no_round if dtype == "float32" else plain.bf16_round
    want = [plain.delta_mixer(s.double(), wd, m, eps, ROUND) for s in seqs]
    records = torch.zeros(4, part.record_floats, device="cuda")
    view = SimpleNamespace(records=records)
    fn = lambda x, step: _sum(part.forward(dev(x, TORCH[dtype]), step, view), x.shape[0])
    tol = 4.0 if dtype == "float32" else 3.0
    for _ in range(2):
        records[SLOTS] = 0.0                    # what the cache does when it hands a slot out
        records[1] = float("nan")               # nobody's slot
        for g, ref in zip(run_in_steps(seqs, SLOTS, CUTS, fn), want):
            close(g, ref, dtype, scale=tol)
    assert records[1].isnan().all()
    long = rnd(130, width)
    records[1] = 0.0
    got = run_in_steps([long], [1], [[80, 2, 48]], fn)[0]
    close(got, plain.delta_mixer(long.double(), wd, m, eps, ROUND), dtype, scale=tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,taps", [(4, 2, 12, 20, 3), (3, 3, 130, 33, 2), (2, 1, 64, 200, 4), (2, 2, 7, 9, 6)])
def test_delta_rule_inputs_in_every_launch_shape(dtype, H, G, dk, dv, taps):
    """Requests whose tokens begin and end inside the runs of tokens that a warp takes; the same bits and the same
    tails from every shape, and a step so large that the launcher takes the shape for many tokens itself."""
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(dk)
    rnd = _rounded(gen, dtype)
    lens = [1, 5, 2, 1, 9, 700, 3, 2]
    n, cols, chans = sum(lens), 2 * G * dk + H * dv + H, 2 * G * dk + H * dv
    proj, a = dev(rnd(n, cols), TORCH[dtype]), dev(rnd(n, H * dk), TORCH[dtype])
    conv, a_log, bias = 0.5 * torch.randn(chans, taps, generator=gen), torch.randn(H, generator=gen), torch.randn(H * dk, generator=gen)
    floats, tail_off = ops.delta_record_floats(H, G, dk, dv, taps)
    start = torch.randn(9, floats, generator=gen)
    slots = [3, 8, 1, 0, 5, 2, 7, 4]
    step = fake_step(lens, slots, [4] * len(lens))
    kw = dict(dtype=TORCH[dtype], q_off=0, k_off=G * dk, v_off=2 * G * dk, b_off=chans, a_off=0, heads=H, kv_heads=G, key_dim=dk,
              value_dim=dv, unit_eps=1e-6, q_scale=dk ** -0.5, channel_a=a)
    got = []
    for shape in (1, 2, 3, 0):
        records = dev(start)
        got.append((*ops.delta_prepare(proj, dev(conv), dev(a_log), dev(bias), records, step.tok_req, step.req_q_start, step.req_q_len,
                                       step.req_slot, step.err, shape=shape, **kw), records))
    assert step.err.tolist()[0] == 0
    for other in got[1:]:
        assert all(torch.equal(x, y) for x, y in zip(got[0], other))
    x = proj.cpu().double()
    at = 0
    for n_r, slot in zip(lens, slots):          # against the plain functions, continuing from the tails
        past = start[slot, tail_off:].view(taps - 1, chans).double()
        y = plain.short_conv(torch.cat([past, x[at:at + n_r, :chans]]), conv.double())[taps - 1:]
        q = plain.unit_vector(y[:, :G * dk].reshape(n_r, G, dk)) * dk ** -0.5
        k = plain.unit_vector(y[:, G * dk:2 * G * dk].reshape(n_r, G, dk))
        g = plain.channel_decay(a[at:at + n_r].cpu().double(), a_log.double(), bias.double())
        for want, have in zip((q, k, y[:, 2 * G * dk:].reshape(n_r, H, dv), torch.sigmoid(x[at:at + n_r, chans:]), g), got[3]):
            close(have[at:at + n_r], want, "float32")
        at += n_r


def test_channel_decays_each_act_on_their_own_row():
    """One written key channel per token and decays of exactly 0, 1/2 and 1: what is read back names the row."""
    from tokamak_b200.csrc import ops
    dk, dv, H = 8, 5, 2
    q, k = torch.zeros(4, H, dk), torch.zeros(4, H, dk)
    v = torch.randn(4, H, dv, generator=torch.Generator().manual_seed(0))
    k[0, :, 3] = 1.0
    k[1, :, 5] = 1.0
    q[2, :, 3], q[2, :, 5] = 1.0, 10.0
    q[3, :, 3], q[3, :, 5] = 1.0, 10.0
    g = torch.ones(4, H, dk)
    g[2, :, 3] = 0.5
    g[3, 0, 5], g[3, 1, 3] = 0.0, 0.0
    beta = torch.ones(4, H)
    step = fake_step([4], [0], [0])
    rec = torch.zeros(1, H * dk * dv, device="cuda")
    o = ops.delta_scan(dev(q), dev(k), dev(v), dev(beta), dev(g), rec, step.req_q_start, step.req_q_len, step.req_slot, step.err).cpu()
    # token 2 and 3 write nothing (k = 0) and read rows 3 and 5
    assert torch.allclose(o[2], 0.5 * v[0] + 10.0 * v[1]) and torch.allclose(o[3, 0], 0.5 * v[0, 0]) and torch.allclose(o[3, 1], 10.0 * v[1, 1])
    ref, S = plain.delta_recurrence(*(t.double() for t in (q, k, v, beta, g)))
    close(o, ref, "float32")
    close(rec.view(H, dk, dv), S, "float32")


# ======================================================================= experts

@pytest.mark.parametrize("experts,identity,top,count,keep,shared", [
    (6, 2, 3, 4, 2, 1), (11, 5, 3, 4, 2, 0), (9, 0, 2, 3, 1, 2), (5, 1, 6, 1, 1, 1), (1, 1, 1, 2, 1, 0), (60, 68, 8, 16, 5, 3), (3, 300, 7, 3, 3, 1)])
def test_router_over_all_outputs_with_groups_identity_and_shared_experts(experts, identity, top, count, keep, shared):
    """The chosen experts and weights of every token, tokens whose best group holds identity experts only, negative
    choice scores, the layout of the pairs and the pairs that have no row."""
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(experts + identity)
    n, width, total = 500, 40, experts + identity
    h = torch.randn(n, width, generator=gen)
    w = {"router": 0.5 * torch.randn(total, width, generator=gen), "correction": 0.2 * torch.randn(total, generator=gen) - 1.0}
    sg = torch.randn(1, width, generator=gen)
    chosen, weights, margin = plain.route(h.double(), _doubles(w), {"experts": experts, "identity": identity, "top": top,
                                                                    "groups": {"count": count, "keep": keep}})
    router = torch.cat([w["router"], sg]) if shared else w["router"]
    r = ops.moe_route(dev(h), dev(router), dev(w["correction"]), top=top, n_groups=count, keep=keep, padded=True,
                      kind="softmax_all", group_score="best", normalize=True, identity=identity, shared=shared)
    got, gw = r.chosen.cpu().long(), r.weights.cpu().double()
    clear = margin > 1e-6
    assert clear.float().mean() > 0.9
    is_id = chosen >= experts
    assert torch.equal(got[clear, :top], chosen.masked_fill(is_id, -1)[clear])
    assert (gw[:, :top] - weights.masked_fill(is_id, 0.0))[clear].abs().max() < 1e-5
    if identity:
        own = (weights * is_id).sum(-1)
        assert (r.identity_weight.cpu()[:, 0].double() - own)[clear].abs().max() < 1e-5
    if shared:
        gate = torch.sigmoid(h.double() @ sg.double().T)
        assert torch.equal(got[:, top:], torch.arange(experts, experts + shared).expand(n, shared))
        assert (gw[:, top:] - gate).abs().max() < 1e-5
    # the layout: every pair with a row has one of its own, in a tile of its expert
    pair_row, tile = r.pair_row.cpu(), r.tile_expert.cpu()
    flat = got.reshape(-1)
    assert torch.equal(pair_row >= 0, flat >= 0)
    rows = pair_row[flat >= 0].long()
    assert len(set(rows.tolist())) == len(rows) and torch.equal(tile[rows // ops.moe_pad_rows()].long(), flat[flat >= 0])
    listed = r.order.cpu()[:len(rows)].long()
    assert torch.equal(listed.sort().values, (flat >= 0).nonzero()[:, 0]) and (flat[listed].diff() >= 0).all()


def _moe_weights(gen, dtype, width, ff, experts, identity, shared):
    rnd = _rounded(gen, dtype)
    s = 1.5 / width ** 0.5
    w = {"router": 3 * rnd(experts + identity, width, std=s), "correction": 0.05 * torch.randn(experts + identity, generator=gen)}
    names = [(f"e{e}.", ff) for e in range(experts)] + ([("shared.", shared)] if shared else [])
    for p, f in names:
        w[p + "gate"], w[p + "up"] = rnd(f, width, std=s), rnd(f, width, std=s)
        w[p + "down"] = rnd(width, f, std=1.5 / f ** 0.5)
    if shared:
        w["shared.sg"] = rnd(1, width, std=s)
    return w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,ff,experts,identity,top,count,keep,shared", [
    (70, 48, 40, 6, 2, 3, 4, 2, 24), (1, 64, 64, 4, 4, 2, 2, 1, 64), (2, 128, 96, 7, 1, 2, 4, 3, 200), (300, 54, 30, 5, 1, 2, 3, 2, 70),
    (900, 136, 64, 13, 3, 5, 4, 3, 128), (5, 64, 128, 8, 0, 2, 1, 1, None), (40, 96, 100, 3, 3, 5, 2, 2, None)])
def test_experts_with_identity_and_shared_ones_through_the_feed_forward(dtype, n, width, ff, experts, identity, top, count, keep, shared):
    from tokamak_b200.parts.base import FEED_FORWARDS, SumBranch
    from tokamak_b200.parts.feedforward import MoESpec
    gen = torch.Generator().manual_seed(n + ff)
    w = _moe_weights(gen, dtype, width, ff, experts, identity, shared)
    h = _rounded(gen, dtype)(n, width)
    mlp = {"router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": count, "keep": keep}},
           "shared": None if shared is None else {"ff": shared}}
    margins = []
    want = plain.mixture(h.double(), _doubles(w), mlp, plain.no_round, margins)
    part = _part(FEED_FORWARDS, MoESpec(hidden_size=width, intermediate_size=ff, num_experts=experts, top=top, num_groups=count,
                                        keep_groups=keep, router="softmax_all", normalize=True, group_score="best",
                                        identity=identity, shared_size=shared, pad_inner=True), w, dtype)
    if dtype == "bfloat16" and width % 8 == 0:
        assert part.w_first is not None                 # the tensor cores' grouped product, or the small steps' kernel
    step = fake_step([n], [0], [0])
    x = dev(h, TORCH[dtype])
    clear = margins[0] > 1e-5
    got = part.forward(x, step)[0]
    close(got[dev(clear)], want[clear], dtype, scale=2.0)
    assert got.isfinite().all() and step.err.tolist()[0] == 0
    # the terms in front of their sum, joined by the kernel of the next norm beside another branch
    terms = part.forward(x, step, combine=False)
    terms = terms if isinstance(terms, tuple) else (terms,)
    assert len(terms) == 1 + (identity > 0)
    from tokamak_b200.csrc import ops
    resid = torch.randn(n, width, generator=gen)
    a = _rounded(gen, dtype)(n, width)
    out, stream = torch.empty(n, width, dtype=TORCH[dtype], device="cuda"), dev(resid)
    ops.sum_rmsnorm(stream, (dev(a, TORCH[dtype]), *terms), out, torch.ones(width, device="cuda"), 1e-5)
    sum_ = resid.double() + a.double() + want
    close(stream[dev(clear)], sum_[clear], dtype, scale=2.0)
    settled = dev(resid)
    SumBranch((dev(a, TORCH[dtype]), *terms)).settle(settled)
    assert (settled - stream).abs().max() < 1e-4
    # the result of a token does not depend on the others in the step
    if dtype == "float32":
        pick = torch.arange(0, n, 7)
        assert (part.forward(x[dev(pick)].contiguous(), fake_step([len(pick)], [0], [0]))[0] - got[dev(pick)]).abs().max() < 1e-6


# ======================================================================= whole models

LENGTHS = {"XA": [5, 17, 33, 70, 130, 96, 41, 128], "XB": [1, 7, 31, 64, 100, 143, 52, 90],
           "XC": [3, 40, 77, 150, 64, 110, 25, 95], "XD": [2, 66, 129, 20, 90, 151, 47, 80]}
TAGS = ["XA", "XB", "XC", "XD"]


def requests_for(tag):
    vocab = sc.ALL[tag][0]["vocab"]
    return {f"r{i}": random_tokens(vocab, n, seed=100 * i + n) for i, n in enumerate(LENGTHS[tag])}


def make_core(tag, dtype, max_tokens, max_live=4):
    from tokamak_b200.engine.replay import build_core
    return build_core(folder_of(tag, dtype), dtype, max_tokens, page_size=sc.ALL[tag][2], max_live=max_live)


def replay(tag, dtype, builder, max_tokens, poison=False, max_live=4, **kw):
    from tokamak_b200.engine.replay import run_step
    reqs = requests_for(tag)
    if builder is traces.mixed:
        kw.update(max_tokens=max_tokens, max_live=max_live)
    records, rows = builder(reqs, **kw)
    core = make_core(tag, dtype, max_tokens, max_live)
    results = {}
    for rec in records:
        if poison:
            core.cache.poison_free_pages()
            core.cache.poison_free_state()
        out = run_step(core, rec)
        if out is not None:
            results[rec["step"]] = out
        core.manager.check_invariants()
    assert not core.manager.live_requests()
    assert all(g.num_free == g.num_pages for g in core.manager.kv_groups)
    n = check_rows(results, rows, reqs, folder_of(tag, dtype), dtype, f"{tag}/{dtype}")
    assert n == sum(len(v) for v in rows.values())
    return core


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag", TAGS)
def test_whole_prompts(tag, dtype):
    replay(tag, dtype, traces.whole, max_tokens=192)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag", TAGS)
def test_tail_decoded_one_by_one_across_every_window(tag, dtype):
    replay(tag, dtype, traces.tail_one_by_one, max_tokens=192, tail=70)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag", TAGS)
def test_portions_of_changing_size(tag, dtype):
    replay(tag, dtype, traces.portions, max_tokens=192)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tag", TAGS)
def test_mixed_batches_with_pages_and_slots_used_again(tag, dtype):
    replay(tag, dtype, traces.mixed, max_tokens=384, poison=True, seed=7)
    assert sum(LENGTHS[tag]) > 384


@pytest.mark.parametrize("seed", [1, 2])
@pytest.mark.parametrize("tag,dtype", [("XA", "float32"), ("XB", "bfloat16"), ("XC", "bfloat16"), ("XD", "float32")])
def test_mixed_batches_in_other_orders_with_two_slots(tag, dtype, seed):
    replay(tag, dtype, traces.mixed, max_tokens=320, poison=True, seed=seed, max_live=2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_and_long_decode(dtype):
    """Positions 0, 1, 2 one by one, then 220 more decoded one by one: over many pages that windows give back on
    the way, the states carried through every step."""
    from tokamak_b200.engine.replay import run_trace
    tag = "XA"
    reqs = {"long": random_tokens(sc.ALL[tag][0]["vocab"], 224, seed=5)}
    records, rows = traces.tail_one_by_one(reqs, tail=223)
    results = run_trace(make_core(tag, dtype, 256), records)
    check_rows(results, rows, reqs, folder_of(tag, dtype), dtype, f"long/{dtype}")


def test_same_logits_however_cut_float32():
    from tokamak_b200.engine.replay import run_trace
    tag = "XB"
    reqs = requests_for(tag)
    got = {}
    for name, builder in (("whole", traces.whole), ("portions", traces.portions)):
        records, rows = builder(reqs)
        res = run_trace(make_core(tag, "float32", 192), records)
        got[name] = {rp: res[s][i] for s in rows for i, rp in enumerate(rows[s])}
    for rp, a in got["whole"].items():
        b = got["portions"][rp]
        assert np.abs(a - b).max() <= 2e-5 * max(1.0, np.abs(a).max()), rp


@pytest.mark.parametrize("tag", TAGS)
def test_residual_stream_after_every_layer_run_float32(tag):
    """Layer run by layer run (a looped layer counts every time): the stream with what the block leaves pending
    added, against the plain implementation."""
    from tokamak_b200.engine.step import StepEntry
    from tokamak_b200.parts.base import NormedSum, SumBranch, sum_parts
    core = make_core(tag, "float32", 64)
    caught = []

    def joined(resid, pending):
        u = resid.double()
        if isinstance(pending, SumBranch):
            v = torch.zeros_like(resid)
            pending.settle(v)
            return u + v.double()
        if isinstance(pending, NormedSum):
            for b in (pending.first, pending.second):
                u = u + plain.unit_rms(sum_parts(b.x).double(), b.eps) * b.weight.double()
            return u
        return u + sum_parts(pending).double()

    for block in core.model.blocks.values():
        def wrapped(resid, pending, step, view, next_norm=None, fwd=block.forward):
            r, p = fwd(resid, pending, step, view)
            caught.append(joined(r, p).cpu())
            return r, p
        block.forward = wrapped
    toks = random_tokens(sc.ALL[tag][0]["vocab"], 40, seed=9)
    core.step.run([StepEntry("a", toks, [39])])
    cfg, w = plain.load_folder(folder_of(tag, "float32"))
    want = []
    plain.forward(cfg, w, toks, layers_out=want)
    assert len(caught) == len(want) == len(core.model.spec.schedule)
    for i, got in enumerate(caught):
        err = (got - want[i]).abs().max().item()
        assert err <= 2e-4 * max(1.0, want[i].abs().max().item()), f"layer run {i} is off by {err:.3e}"


@pytest.mark.parametrize("tag", ["XA", "XB"])
def test_greedy_generation_through_the_entry_point_float32(tag):
    """LLM.generate with its scheduler: prompts in portions beside decoding requests, fewer slots
    than requests, a pool that is used again; the tokens are the plain implementation's."""
    from tokamak_b200 import LLM, SamplingParams
    folder = folder_of(tag, "float32")
    llm = LLM(folder, dtype="float32", block_size=sc.ALL[tag][2], max_seq_len=128, kv_pool_tokens=256,
              prefill_chunk=24, max_num_batched_tokens=40, max_batch_size=3)
    vocab = sc.ALL[tag][0]["vocab"]
    prompts = [random_tokens(vocab, n, seed=7 * n + 1) for n in (5, 33, 1, 61, 18)]
    outs = llm.generate(prompt_token_ids=prompts, sampling_params=SamplingParams(temperature=0.0, max_new_tokens=10))
    assert llm.last_stats["mixed_steps"] > 0
    cfg, w = plain.load_folder(folder)
    for p, o in zip(prompts, outs):
        assert o.output_token_ids == plain.greedy_generate(cfg, w, p, 10), len(p)


def test_preemption_is_invisible_in_greedy_tokens_float32():
    """A pool so small that requests are evicted and recomputed: states start over with the request, and the tokens
    are those of a large pool and of the plain implementation."""
    from tokamak_b200 import LLM, SamplingParams
    tag = "XC"                                   # windows of 33 to 80: the pool of the longest runs out
    folder = folder_of(tag, "float32")
    prompts = [random_tokens(sc.ALL[tag][0]["vocab"], n, seed=3 * n) for n in (40, 55, 48, 60)]
    params = SamplingParams(temperature=0.0, max_new_tokens=30)
    got = {}
    for pool in (1024, 192):
        llm = LLM(folder, dtype="float32", block_size=8, max_seq_len=96, kv_pool_tokens=pool, max_batch_size=4)
        got[pool] = [o.output_token_ids for o in llm.generate(prompt_token_ids=prompts, sampling_params=params)]
        assert (llm.last_stats["preemptions"] > 0) == (pool == 192)
    assert got[192] == got[1024]
    cfg, w = plain.load_folder(folder)
    assert got[1024][1] == plain.greedy_generate(cfg, w, prompts[1], 30)


def test_greedy_generation_bfloat16_with_graphs_picks_top_tokens():
    """Decode steps replayed from CUDA graphs (every part of the design declares them safe): the tokens are
    those of the same engine with every step laid out by the host, and nearly the plain implementation's best
    for their prefix."""
    from tokamak_b200 import LLM, SamplingParams
    tag = "XC"
    folder = folder_of(tag, "bfloat16")
    llm = LLM(folder, dtype="bfloat16", block_size=sc.ALL[tag][2], max_seq_len=128, max_batch_size=4)
    assert llm.core.model.graph_safe()
    prompts = [random_tokens(sc.ALL[tag][0]["vocab"], n, seed=n) for n in (9, 40, 70)]
    params = SamplingParams(temperature=0.0, max_new_tokens=12)
    outs = llm.generate(prompt_token_ids=prompts, sampling_params=params)
    replays = llm.core.step.graph_replays
    assert replays > 0
    llm.plain_steps = True
    slow = llm.generate(prompt_token_ids=prompts, sampling_params=params)
    assert llm.core.step.graph_replays == replays
    assert [o.output_token_ids for o in outs] == [o.output_token_ids for o in slow]
    near = total = 0
    for p, o in zip(prompts, outs):
        seq = list(p)
        for tok in o.output_token_ids:
            logits = _truth(str(folder), tuple(seq))[0][-1]
            near += bool(logits[tok] >= logits.max() - 0.1 * logits.std())
            total += 1
            seq.append(tok)
    assert near >= 0.8 * total


def test_trace_run_program_on_this_design(tmp_path):
    tag, dtype = "XD", "float32"
    reqs = {k: v for k, v in list(requests_for(tag).items())[:4]}
    records, rows = traces.mixed(reqs, max_tokens=256, seed=3)
    folder = folder_of(tag, dtype)
    out = tmp_path / "out"
    proc = subprocess.run(
        [sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype,
         "--out", str(out), "--max-tokens", "256", "--page-size", "8"],
        input="".join(json.dumps(r) + "\n" for r in records), text=True, capture_output=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.split() == [w for r in records for w in ("done", str(r["step"]))]
    vocab = sc.ALL[tag][0]["vocab"]
    results = {s: np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, vocab) for s in rows}
    check_rows(results, rows, reqs, folder, dtype, "trace_run")


def test_generation_from_the_command_line(capsys):
    from tokamak_b200.cli import main
    folder = folder_of("XA", "float32")
    argv = ["--model", str(folder), "--dtype", "float32", "--prompt-len", "21", "--temperature", "0",
            "--max-new-tokens", "9", "--ignore-eos", "--block-size", "16", "--max-seq-len", "64", "--kv-pool-tokens", "256"]
    assert main(argv) == 0
    first = capsys.readouterr().out
    assert main(argv) == 0
    assert capsys.readouterr().out == first and first.strip()
