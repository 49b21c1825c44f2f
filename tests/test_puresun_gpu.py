"""The Puresun design on the GPU: every mechanism's kernels against the plain implementation, then whole
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

import puresun_configs as pc
import traces
from helpers import assert_logits_close, random_tokens
from plain import puresun_plain as plain

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
_TMP = []


@functools.lru_cache(maxsize=None)
def folder_of(tag: str, dtype: str) -> Path:
    tmp = tempfile.TemporaryDirectory(prefix=f"ps_{tag}_{dtype}_")
    _TMP.append(tmp)
    return Path(pc.write_folder(tmp.name, tag, dtype))


@functools.lru_cache(maxsize=None)
def _truth(folder: str, tokens: tuple):
    """Logits of the whole sequence, and for every position how close any router came to another choice at
    or before it (a choice made otherwise early in a sequence reaches later positions through the keys)."""
    cfg, w = plain.load_folder(folder)
    margins = []
    logits = plain.forward(cfg, w, list(tokens), margins_out=margins)
    risk = torch.stack(margins).min(0).values.cummin(0).values if margins else torch.full((len(tokens),), math.inf)
    return logits, risk


# bfloat16: a row is judged against what rounding alone costs in its request (the plain implementation
# rounding at every product's input and output): the level is the worst row of the request, the limit four
# times that and never below the level of a well-conditioned row.  A wrong key, pair row, expert or vector moves a
# row by about its spread.  So does a router that rounding tips elsewhere than in the plain implementation: the
# few rows beyond the limit that have a router within CLOSE of another choice, at or before them, are let through,
# counted.
BF16_FLOOR_RMS, BF16_FLOOR_MAX, BF16_TIMES = 0.05, 0.2, 4.0
CLOSE, TIPPED_ROWS, TIPPED_SHARE = 0.05, 2, 0.06


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


def fake_step(q_lens, slots, starts, tokens=None):
    """What a kernel reads of a step: requests of ``q_lens`` tokens in ``slots``, continuing at ``starts``."""
    tok_req, pos, q_start = [], [], []
    at = 0
    for r, (n, s) in enumerate(zip(q_lens, starts)):
        q_start.append(at)
        tok_req += [r] * n
        pos += list(range(s, s + n))
        at += n
    return SimpleNamespace(tok_req=i32(tok_req), positions=i32(pos), req_q_start=i32(q_start), req_q_len=i32(q_lens),
                           req_slot=i32(slots), req_kv_len=i32([s + n for s, n in zip(starts, q_lens)]),
                           err=torch.zeros(4, dtype=torch.int32, device="cuda"), max_q_len=max(q_lens), n_tokens=at,
                           scratch={}, token_ids=i32(tokens if tokens is not None else [0] * at),
                           decode_items=i32([s for s, n in zip(q_start, q_lens) if n == 1]),
                           prefill_items=i32([s + j for s, n in zip(q_start, q_lens) if n > 1 for j in range(n)]),
                           prefill_tiles=i32([x for r, n in enumerate(q_lens) if n > 1 for t in range(-(-n // 64)) for x in (r, t)]),
                           max_kv_len=max(s + n for s, n in zip(starts, q_lens)))


def run_in_steps(seqs, slots, cuts, fn):
    """Feed sequences (``[T, ...]`` each, one per request) through ``fn(rows of the step, step)`` cut into steps:
    ``cuts[r]`` lists request r's portion sizes, step by step (0: the request sits the step out).  Returns
    the outputs put together again per request."""
    outs = [[] for _ in seqs]
    fed = [0] * len(seqs)
    for s in range(max(len(c) for c in cuts)):
        live = [r for r in range(len(seqs)) if s < len(cuts[r]) and cuts[r][s] > 0]
        step = fake_step([cuts[r][s] for r in live], [slots[r] for r in live], [fed[r] for r in live])
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


CUTS = [[5, 1, 1, 0, 2, 7, 1], [1, 1, 3, 9, 0, 2], [16, 1, 0, 0, 1, 1, 2]]      # the second step is single tokens only
SLOTS = [2, 0, 3]


# ======================================================================= mechanisms alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,vocab,buckets,mul_prev,mul_cur", [(48, 77, 31, 7, 13), (54, 90, 1009, 7368787, 15485863),
                                                                   (1028, 40, 5, 0, 1), (7, 40, 1, 3, 5)])
def test_bigram_rows_with_the_previous_token_carried_over_steps(dtype, width, vocab, buckets, mul_prev, mul_cur):
    """Three requests fed in steps of unequal portions, single tokens among them, now and then sitting a step out:
    the first token takes the last pair row, every other the row of its pair, across portions too; a slot nobody
    uses is left alone, and one that is used again starts anew whatever it holds."""
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(width)
    w = {"embed": torch.randn(vocab, width, generator=gen).to(TORCH[dtype]),
         "bigram": torch.randn(buckets + 1, width, generator=gen).to(TORCH[dtype])}
    table, pairs = dev(w["embed"]), dev(w["bigram"])
    last = torch.full((4, 1), -(1 << 30), dtype=torch.int32, device="cuda")
    bg = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    for turn in range(2):                        # the second turn uses the slots again
        seqs = [torch.randint(0, vocab, (sum(c),), generator=gen) for c in CUTS]
        kept = []

        def fn(rows, step):
            step.token_ids = rows.to("cuda", torch.int32)
            resid = torch.empty(len(rows), width, device="cuda")
            keep = torch.empty_like(resid) if step.n_tokens % 2 else None
            ops.embed_bigram(table, pairs, last, step, resid, mul_prev=mul_prev, mul_cur=mul_cur, scale=1.0, keep=keep)
            if keep is not None:
                kept.append(torch.equal(keep, resid))
            return resid
        for got, toks in zip(run_in_steps(seqs, SLOTS, CUTS, fn), seqs):
            close(got, plain.embedding({k: t.double() for k, t in w.items()}, toks.tolist(), bg), "float32")
        assert kept and all(kept)
        assert [last[s].item() for s in SLOTS] == [int(x[-1]) for x in seqs] and last[1].item() == -(1 << 30)


def test_bigram_kernel_reports_tokens_it_cannot_look_up():
    from tokamak_b200.csrc import ops
    table, pairs = torch.ones(5, 8, device="cuda"), torch.ones(4, 8, device="cuda")
    for toks, held, start in (([2, 9, 1], 0, 0), ([1, -1, 1], 0, 0), ([1, 2, 1], 77, 3)):
        last = torch.full((1, 1), held, dtype=torch.int32, device="cuda")
        step = fake_step([3], [0], [start], toks)
        resid = torch.full((3, 8), 7.0, device="cuda")
        ops.embed_bigram(table, pairs, last, step, resid, mul_prev=1, mul_cur=1)
        assert step.err.tolist()[0] == 1 and (resid != 7.0).all()


def _weighted(gen, n, width, top, dtype, listed):
    from tokamak_b200.csrc import ops
    rows = n * top + 5
    y = torch.randn(rows if listed else n * top, width, generator=gen).to(dtype)
    weights = torch.rand(n, top, generator=gen)
    pair_row = torch.randperm(rows, generator=gen)[:n * top].int() if listed else None
    at = pair_row.long() if listed else torch.arange(n * top)
    want = (weights.double().reshape(-1, 1) * y.double()[at]).view(n, top, width).sum(1)
    return ops.WeightedRows(dev(y), dev(weights), dev(pair_row) if listed else None), want


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,n", [(42, 5), (48, 11), (256, 3), (1100, 300), (4096, 9), (8200, 2)])
def test_sum_of_several_branches_and_its_norm(dtype, width, n):
    """Every kind of branch (rows, partial sums, weighted rows with and without a list, in both types), kept rows
    and a vector for every token, alone and together; with a list of rows the stream stays as it is."""
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(width + n)
    x = torch.randn(n, width, generator=gen) * 2.0
    w = 1.0 + 0.2 * torch.randn(width, generator=gen)
    rows = torch.randn(n, width, generator=gen).to(TORCH[dtype])
    parts = torch.randn(3, n, width, generator=gen)
    w16, want16 = _weighted(gen, n, width, 3, torch.bfloat16, True)
    w32, want32 = _weighted(gen, n, width, 2, torch.float32, False)
    extra, vec = torch.randn(n, width, generator=gen), torch.randn(width, generator=gen)
    close(w16.combine(), want16, "float32")
    close(w32.combine(), want32, "float32")
    zero = torch.zeros(n, width, dtype=torch.float64)
    sources = {"rows": (dev(rows), rows.double()), "parts": (dev(parts), parts.double().sum(0)),
               "w16": (w16, want16), "w32": (w32, want32)}
    cases = [((), False, True), ((), True, False), (("rows",), False, False), (("parts", "w16"), True, True),
             (("rows", "w32"), False, True), (("w16", "parts"), False, False), (("w32", "rows"), True, False)]
    pick = [n - 1, 0, n // 2]
    for names, with_extra, with_vec in cases:
        total = x.double() + sum((sources[k][1] for k in names), zero)
        total = total + (extra.double() if with_extra else 0.0) + (vec.double() if with_vec else 0.0)
        want = plain.rms_norm(total, w.double(), 1e-5)
        kw = dict(extra=dev(extra) if with_extra else None, vector=dev(vec) if with_vec else None)
        resid = dev(x.clone())
        out = torch.empty(n, width, dtype=TORCH[dtype], device="cuda")
        ops.sum_rmsnorm(resid, [sources[k][0] for k in names], out, dev(w), 1e-5, **kw)
        close(resid, total, "float32")
        close(out, want, dtype)
        resid = dev(x.clone())
        out = torch.empty(3, width, dtype=TORCH[dtype], device="cuda")
        ops.sum_rmsnorm(resid, [sources[k][0] for k in names], out, dev(w), 1e-5, rows=i32(pick), **kw)
        close(out, want[pick], dtype)
        assert torch.equal(resid.cpu(), x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,d,dr,rank,n_rot", [(3, 16, 8, 24, 8), (4, 8, 12, 16, 6), (2, 32, 64, 96, 64), (1, 4, 7, 300, 2),
                                                   (5, 6, 4, 20, 0)])
def test_latent_rows_with_a_rotated_part_in_halves(dtype, heads, d, dr, rank, n_rot):
    """The cache row [c | rot(k_r)] in the token's page and slot and the query rows, the rotated part turning in
    halves (all of it, its first elements, none of it), from rows and from the sums of a split product."""
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(d * dr + rank)
    n, page, cols_q = 11, 4, heads * (d + dr)
    proj = torch.randn(n, cols_q + rank + dr + 5, generator=gen).to(TORCH[dtype])
    wc = 1 + 0.3 * torch.randn(rank, generator=gen)
    positions = [5, 6, 7, 8, 9, 0, 1, 2, 13, 14, 15]          # three requests: 5 tokens from 5, 3 from 0, 3 from 13
    tok_req, slots = [0] * 5 + [1] * 3 + [2] * 3, [2, 0, 1]
    pages = torch.full((3, 6), -1, dtype=torch.int32)
    pages[2, :3] = torch.tensor([7, 3, 8]); pages[0, :1] = 5; pages[1, :4] = torch.tensor([1, 0, 2, 6])
    pos = torch.tensor(positions)
    freq = torch.tensor([300.0 ** (-2.0 * i / n_rot) for i in range(n_rot // 2)], dtype=torch.float32)
    rope = ops.rope_table(dev(pos.int()), dev(freq)) if n_rot else None
    cache = torch.zeros(9, 1, page, rank + dr, dtype=TORCH[dtype], device="cuda")
    q_abs = torch.randn(heads, n, rank, generator=gen)
    err = torch.zeros(4, dtype=torch.int32, device="cuda")
    args = (dev(pos.int()), i32(tok_req), i32(slots), dev(pages), err)
    kw = dict(kv_off=cols_q, rank=rank, rot=dr, kv_norm_w=dev(wc), eps=1e-5, table=rope, q_abs=dev(q_abs), q_off=0,
              q_head_cols=d + dr, q_rot_off=d, halves=True)
    q_lat, _ = ops.latent_prepare(dev(proj), cache, *args, **kw)
    assert err.tolist()[0] == 0
    x = proj.double()
    turn = (lambda t: plain.rotate_halves(t, pos, n_rot, 300.0)) if n_rot else (lambda t: t)
    c = plain.rms_norm(x[:, cols_q:cols_q + rank], wc.double(), 1e-5)
    want = torch.cat([c, turn(x[:, None, cols_q + rank:cols_q + rank + dr])[:, 0]], 1)
    for t in range(n):
        close(cache[pages[slots[tok_req[t]], positions[t] // page].item(), 0, positions[t] % page], want[t], dtype, scale=2.0)
    close(q_lat[..., :rank], q_abs.transpose(0, 1), "float32")
    close(q_lat[..., rank:], turn(x[:, :cols_q].reshape(n, heads, d + dr)[..., d:]), "float32", scale=2.0)
    cache2 = torch.zeros_like(cache)
    split = dev(torch.stack([proj.float() * 0.5, proj.float() * 0.5]))
    q_lat2, _ = ops.latent_prepare(split, cache2, *args, **kw)
    assert torch.equal(q_lat2, q_lat) and torch.equal(cache2, cache)


def _part(registry, spec, weights, dtype, prefix="m."):
    from tokamak_b200.parts.base import Runtime
    cls = registry.get(spec.kind)
    tensors = {}
    for name, req in cls.expected_tensors(spec, prefix).items():
        t = weights[name[len(prefix):]]
        assert tuple(t.shape) == tuple(req.shape), name
        tensors[name] = dev(t, TORCH[dtype] if req.role == "matrix" else torch.float32)
    return cls(spec, prefix, tensors, Runtime(device=torch.device("cuda"), dtype=TORCH[dtype]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,dr,dv,rank,window,page", [(3, 16, 8, 20, 24, 9, 4), (4, 32, 32, 48, 64, 16, 16), (2, 12, 4, 8, 18, 1, 8),
                                                        (18, 8, 16, 24, 80, 70, 16), (5, 16, 16, 16, 48, 64, 8), (1, 24, 8, 12, 32, 500, 4)])
def test_latent_attention_with_keys_that_stand_out_at_the_windows_edges(dtype, H, d, dr, dv, rank, window, page):
    """The whole mixer over its cache: one marked key and marked queries around the two edges of its window (the
    last position that sees it, the first that does not), at page borders, right behind it and far away.  The
    marked pair's score beats every other, so that a key that is lost or seen too long moves the row by its whole
    spread (which is checked in the oracle).  Once as a whole prompt, then in portions down to two tokens beside
    another request, then the marked tokens decoded one by one."""
    from tokamak_b200.cache.device import KVView
    from tokamak_b200.parts.base import MIXERS
    from tokamak_b200.parts.latent import LatentAttentionSpec
    from tokamak_b200.parts.position import RopeHalvesSpec
    gen = torch.Generator().manual_seed(H * 100 + rank)
    width, T, eps, key_at = 72, 150, 1e-5, 19
    rnd = lambda *s, std: (torch.randn(*s, generator=gen) * std).to(TORCH[dtype]).float()
    w = {"q": rnd(H * (d + dr), width, std=0.1), "dkv": rnd(rank + dr, width, std=0.2), "dkv.norm": 1 + 0.1 * torch.randn(rank, generator=gen),
         "uk": rnd(H * d, rank, std=0.2), "uv": rnd(H * dv, rank, std=0.3), "g": rnd(H * dv, width, std=0.1),
         "o": rnd(width, H * dv, std=0.2)}
    # the first channel marks keys, the second one queries: the mark puts the latent along its first element and
    # the queries along what W_uk makes of it
    w["dkv"][:, 0], w["q"][:, 1] = 0.0, 0.0
    w["dkv"][0, 0] = 6.0
    for h in range(H):
        col = w["uk"][h * d:(h + 1) * d, 0]
        w["q"][h * (d + dr):h * (d + dr) + d, 1] = (0.75 * col / col.norm() ** 2).to(TORCH[dtype]).float()
    scale = 1.5
    queries = sorted({p for p in (key_at, key_at + 1, key_at + window - 2, key_at + window - 1, key_at + window, key_at + window + 1,
                                  4 * page, 4 * page - 1, T - 1) if key_at <= p < T})
    seqs = [rnd(T, width, std=0.5), rnd(77, width, std=0.5)]
    for s in seqs:
        s[:, :2] = 0.0
    seqs[0][key_at, 0] = 8.0
    seqs[0][queries, 1] = 6.0
    m = {"heads": H, "dim": d, "rot_dim": dr, "vdim": dv, "kv_rank": rank, "scale": scale, "rot": {"base": 200.0, "dims": dr},
         "mask": {"size": window}}
    wd = {k: t.double() for k, t in w.items()}
    want = [plain.latent_attention(s.double(), wd, m, eps, torch.arange(len(s))) for s in seqs]
    for edge, other in ((key_at + window - 1, window - 1), (key_at + window, window + 1)):
        if edge in queries and other > 0:          # a window that is one token off would show
            off = plain.latent_attention(seqs[0].double(), wd, {**m, "mask": {"size": other}}, eps, torch.arange(T))
            assert (off[edge] - want[0][edge]).abs().max() > 0.3 * want[0].std(), (edge, other)
    part = _part(MIXERS, LatentAttentionSpec(hidden_size=width, num_heads=H, head_dim=d, v_head_dim=dv, kv_rank=rank,
                                             softmax_scale=scale, norm_eps=eps, rot_dim=dr,
                                             position=RopeHalvesSpec(dr, 200.0), window=window, gate=True), w, dtype)
    order = torch.randperm(64, generator=gen)
    table = torch.full((4, 40), -1, dtype=torch.int32)
    table[2, :-(-T // page)], table[0, :-(-77 // page)] = order[:-(-T // page)].int(), order[-(-T // page):-(-T // page) - (-77 // page)].int()

    def run(cuts):
        cache = torch.zeros(64, 1, page, rank + dr, dtype=TORCH[dtype], device="cuda")
        view = KVView(cache, cache[..., :rank], dev(table), page, window)
        return run_in_steps(seqs, [2, 0], cuts, lambda rows, step: torch.as_tensor(
            part.forward(dev(rows, TORCH[dtype]), step, view)).float().reshape(-1, rows.shape[0], width).sum(0))

    tol = 3.0 if dtype == "float32" else 6.0
    splits = [[T], [77]], [[7, 2, 30, 2, 64, 3, 2, T - 110], [2, 40, 0, 2, 2, 31]]
    # up to the first marked query at once, then every token alone
    ones = [[key_at - 1] + [1] * (T - key_at + 1), [40, 0, 1, 2] + [1] * 34]
    for cuts in (*splits, ones):
        for got, ref in zip(run(cuts), want):
            close(got, ref, dtype, scale=tol)


@pytest.mark.parametrize("experts,top", [(6, 2), (16, 1), (5, 5), (300, 7), (1, 1)])
def test_softmax_router_over_the_chosen_experts_only(experts, top):
    """The largest logits are chosen, their weights are the softmax over them alone, also where logits are large."""
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(experts * 10 + top)
    n, width = 64, 40
    h, router = torch.randn(n, width, generator=gen) * 2.0, torch.randn(experts, width, generator=gen)
    h[3] *= 40.0                                 # logits in the hundreds
    got = ops.moe_route(dev(h), dev(router), None, top=top, kind="softmax")
    idx, weight = plain.route(h.double(), router.double(), top)
    mine, mine_w = got.chosen.cpu().long(), got.weights.cpu().double()
    assert torch.equal(mine.sort(-1).values, idx.sort(-1).values)
    assert (mine_w.gather(1, mine.argsort(-1)) - weight.gather(1, idx.argsort(-1))).abs().max() < 2e-4
    assert (mine_w.sum(-1) - 1.0).abs().max() < 1e-5


def _experts(gen, n, width, ff, experts, dtype):
    rnd = lambda *s, std=1.0: (torch.randn(*s, generator=gen) * std).to(TORCH[dtype]).float()
    w = {"router": rnd(experts, width, std=0.4)}
    for e in range(experts):
        w[f"e{e}.up"], w[f"e{e}.down"] = rnd(ff, width, std=width ** -0.5), rnd(width, ff, std=ff ** -0.5)
    return rnd(n, width), w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,ff,experts,top", [(70, 48, 40, 6, 2), (1, 64, 72, 4, 1), (300, 30, 130, 9, 4), (700, 136, 104, 9, 3),
                                                    (5, 256, 320, 16, 1), (3, 64, 96, 3, 3), (2, 520, 1088, 8, 2), (8, 72, 8, 40, 1)])
def test_ungated_experts_through_the_feed_forward(monkeypatch, dtype, n, width, ff, experts, top):
    """The part as the model uses it, with the weighted sum and with the rows in front of it: the plain kernels
    (float32, odd sizes), the grouped product on pairs of SMs with the activation in its epilogue, and the
    kernels for few tokens; a token's result is the same bit for bit whatever else is in the step."""
    from tokamak_b200.csrc import ops
    from tokamak_b200.parts.base import FEED_FORWARDS
    from tokamak_b200.parts.feedforward import MoESpec
    gen = torch.Generator().manual_seed(n + width)
    h, w = _experts(gen, n, width, ff, experts, dtype)
    part = _part(FEED_FORWARDS, MoESpec(hidden_size=width, intermediate_size=ff, num_experts=experts, top=top, correction=False,
                                        gated=False, router="softmax", activation="relu2"), w, dtype)
    assert (part.w_first is not None) == (dtype == "bfloat16" and width % 8 == 0 and ff % 8 == 0)
    step = SimpleNamespace(err=torch.zeros(4, dtype=torch.int32, device="cuda"))
    mlp = {"router": {"experts": experts, "top": top}}
    want = plain.mixture(h.double(), {k: t.double() for k, t in w.items()}, mlp,
                         plain.bf16_round if dtype == "bfloat16" else plain.no_round)
    x = dev(h, TORCH[dtype])
    for pairs in (0, 8, 64):                     # the bound up to which the kernels for few tokens are preferred
        monkeypatch.setattr(ops, "MOE_SMALL_PAIRS", pairs)
        got = part.forward(x, step)
        assert got.shape == (1, n, width) and got.dtype == torch.float32
        close(got[0], want, dtype, scale=2.0)
        rows = part.forward(x, step, combine=False)
        assert isinstance(rows, ops.WeightedRows) and torch.equal(rows.combine(), got[0])
        pick = torch.randperm(n, generator=gen)[:max(1, n // 3)]
        if (n * top <= pairs) == (len(pick) * top <= pairs):       # the same kernels for both steps
            assert torch.equal(part.forward(x[pick.to("cuda")].contiguous(), step)[0].cpu(), got[0].cpu()[pick])
    assert step.err.tolist()[0] == 0


@pytest.mark.parametrize("activation", ["silu", "gelu_tanh"])
def test_other_activations_of_ungated_experts(activation):
    from tokamak_b200.csrc import ops
    gen = torch.Generator().manual_seed(3)
    for dtype, n in (("float32", 9), ("bfloat16", 4), ("bfloat16", 90)):
        h, w = _experts(gen, n, 64, 48, 5, dtype)
        up = torch.stack([w[f"e{e}.up"] for e in range(5)])
        down = torch.stack([w[f"e{e}.down"] for e in range(5)])
        idx, weight = plain.route(h.double(), w["router"].double(), 2)
        act = {"silu": torch.nn.functional.silu, "gelu_tanh": lambda z: torch.nn.functional.gelu(z, approximate="tanh")}[activation]
        y = torch.einsum("eft,nef->net", down.transpose(1, 2).double(), act(torch.einsum("eft,nt->nef", up.double(), h.double())))
        want = (weight[..., None] * y.gather(1, idx[..., None].expand(-1, -1, 64))).sum(1)
        x, up, down = (dev(t, TORCH[dtype]) for t in (h, up, down))
        routing = ops.moe_route(x, dev(w["router"]), None, top=2, kind="softmax", padded=dtype == "bfloat16")
        err = torch.zeros(4, dtype=torch.int32, device="cuda")
        close(ops.moe_experts(x, routing, None, up, down, activation), want, dtype, scale=2.0)
        if dtype == "bfloat16":
            close(ops.moe_experts_tc(x, routing, up, down, err, activation, gated=False), want, dtype, scale=2.0)
            if n <= 4:
                close(ops.moe_experts_small(x, routing, up, down, activation, gated=False), want, dtype, scale=2.0)
        assert err.tolist()[0] == 0


# ======================================================================= whole models

LENGTHS = {"SA": [5, 17, 33, 70, 130, 96, 41, 128], "SB": [1, 7, 31, 64, 100, 143, 52, 90],
           "SC": [3, 40, 77, 150, 64, 110, 25, 95], "SD": [2, 66, 129, 20, 90, 151, 47, 80]}
TAGS = ["SA", "SB", "SC", "SD"]


def requests_for(tag):
    vocab = pc.ALL[tag][0]["vocab"]
    return {f"r{i}": random_tokens(vocab, n, seed=100 * i + n) for i, n in enumerate(LENGTHS[tag])}


def make_core(tag, dtype, max_tokens, max_live=4):
    from tokamak_b200.engine.replay import build_core
    return build_core(folder_of(tag, dtype), dtype, max_tokens, page_size=pc.ALL[tag][2], max_live=max_live)


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
@pytest.mark.parametrize("tag,dtype", [("SA", "float32"), ("SB", "bfloat16"), ("SC", "bfloat16"), ("SD", "float32")])
def test_mixed_batches_in_other_orders_with_two_slots(tag, dtype, seed):
    replay(tag, dtype, traces.mixed, max_tokens=320, poison=True, seed=seed, max_live=2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_and_long_decode(dtype):
    """Positions 0, 1, 2 one by one, then 220 more decoded one by one: over many pages that windows give back on
    the way, with the previous token carried through every step."""
    from tokamak_b200.engine.replay import run_trace
    tag = "SA"
    reqs = {"long": random_tokens(pc.ALL[tag][0]["vocab"], 224, seed=5)}
    records, rows = traces.tail_one_by_one(reqs, tail=223)
    results = run_trace(make_core(tag, dtype, 256), records)
    check_rows(results, rows, reqs, folder_of(tag, dtype), dtype, f"long/{dtype}")


def test_same_logits_however_cut_float32():
    from tokamak_b200.engine.replay import run_trace
    tag = "SB"
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
    core = make_core(tag, "float32", 64)
    caught = []
    for block in core.model.blocks.values():
        def wrapped(resid, pending, step, view, fwd=block.forward):
            r, p = fwd(resid, pending, step, view)
            u = r.clone()
            p.settle(u)
            caught.append(u.double().cpu())
            return r, p
        block.forward = wrapped
    toks = random_tokens(pc.ALL[tag][0]["vocab"], 40, seed=9)
    core.step.run([StepEntry("a", toks, [39])])
    cfg, w = plain.load_folder(folder_of(tag, "float32"))
    want = []
    plain.forward(cfg, w, toks, layers_out=want)
    assert len(caught) == len(want) == len(core.model.spec.schedule)
    for i, got in enumerate(caught):
        err = (got - want[i]).abs().max().item()
        assert err <= 2e-4 * max(1.0, want[i].abs().max().item()), f"layer run {i} is off by {err:.3e}"


@pytest.mark.parametrize("tag", ["SA", "SB"])
def test_greedy_generation_through_the_entry_point_float32(tag):
    """LLM.generate with its scheduler: prompts in portions beside decoding requests, fewer slots
    than requests, a pool that is used again; the tokens are the plain implementation's."""
    from tokamak_b200 import LLM, SamplingParams
    folder = folder_of(tag, "float32")
    llm = LLM(folder, dtype="float32", block_size=pc.ALL[tag][2], max_seq_len=128, kv_pool_tokens=256,
              prefill_chunk=24, max_num_batched_tokens=40, max_batch_size=3)
    vocab = pc.ALL[tag][0]["vocab"]
    prompts = [random_tokens(vocab, n, seed=7 * n + 1) for n in (5, 33, 1, 61, 18)]
    outs = llm.generate(prompt_token_ids=prompts, sampling_params=SamplingParams(temperature=0.0, max_new_tokens=10))
    assert llm.last_stats["mixed_steps"] > 0
    cfg, w = plain.load_folder(folder)
    for p, o in zip(prompts, outs):
        assert o.output_token_ids == plain.greedy_generate(cfg, w, p, 10), len(p)


def test_preemption_is_invisible_in_greedy_tokens_float32():
    """A pool so small that requests are evicted and recomputed: the record of the previous token starts over with
    the request, and the tokens are those of a large pool and of the plain implementation."""
    from tokamak_b200 import LLM, SamplingParams
    tag = "SC"                                   # windows of 33 and 80: the pool of the longer one runs out
    folder = folder_of(tag, "float32")
    prompts = [random_tokens(pc.ALL[tag][0]["vocab"], n, seed=3 * n) for n in (40, 55, 48, 60)]
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
    tag = "SC"
    folder = folder_of(tag, "bfloat16")
    llm = LLM(folder, dtype="bfloat16", block_size=pc.ALL[tag][2], max_seq_len=128, max_batch_size=4)
    assert llm.core.model.graph_safe()
    prompts = [random_tokens(pc.ALL[tag][0]["vocab"], n, seed=n) for n in (9, 40, 70)]
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
            near += bool(logits[tok] >= logits.max() - 0.05 * logits.std())
            total += 1
            seq.append(tok)
    assert near >= 0.8 * total


def test_trace_run_program_on_this_design(tmp_path):
    tag, dtype = "SD", "float32"
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
    vocab = pc.ALL[tag][0]["vocab"]
    results = {s: np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, vocab) for s in rows}
    check_rows(results, rows, reqs, folder, dtype, "trace_run")


def test_generation_from_the_command_line(capsys):
    from tokamak_b200.cli import main
    folder = folder_of("SA", "float32")
    argv = ["--model", str(folder), "--dtype", "float32", "--prompt-len", "21", "--temperature", "0",
            "--max-new-tokens", "9", "--ignore-eos", "--block-size", "16", "--max-seq-len", "64", "--kv-pool-tokens", "256"]
    assert main(argv) == 0
    first = capsys.readouterr().out
    assert main(argv) == 0
    assert capsys.readouterr().out == first and first.strip()
