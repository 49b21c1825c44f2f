"""The Puresun design without a GPU: the reader of config.json and its refusals, the tensors it expects, the
order in which looped layers run, what joins the stream in front of them and the caches they get, the sum of
several branches, and the plain implementation's own consistency and its sensitivity to planted mistakes."""

from __future__ import annotations

import copy
from types import SimpleNamespace

import pytest
import torch

import puresun_configs as pc
from plain import puresun_plain as plain
from tokamak_b200.cache.manager import KVPagesNeed, StateNeed
from tokamak_b200.config.model_config import ConfigError
from tokamak_b200.config.registry import architecture_of, supported_architectures
from tokamak_b200.models.decoder import DecoderModel, LayerCall, ModelSpec, StreamInput
from tokamak_b200.parts.base import Runtime, SumBranch

CPU = Runtime(device=torch.device("cpu"), dtype=torch.float32)


def spec_of(raw):
    arch = architecture_of(raw)
    return arch.build_spec(arch.parse(raw))


def cpu_model(raw, tensors=None):
    spec = spec_of(raw)
    names = DecoderModel.expected_tensors(spec)
    return DecoderModel(spec, tensors or {k: torch.zeros(r.shape) for k, r in names.items()}, CPU)


def test_registered_and_parsed():
    assert "Puresun" in supported_architectures()
    arch = architecture_of(pc.PS_A)
    cfg = arch.parse(pc.PS_A)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.logit_softcap, cfg.loop) == (193, 48, 1e-5, 12.0, (1, 3, 2))
    assert (cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur) == (101, 7, 13)
    m = cfg.layers[1].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.window) == (2, 8, 12, 10, 40, 0.25, 40)
    assert (m.rot_dims, m.rot_base) == (12, 500.0)
    assert (cfg.layers[3].mlp.ff, cfg.layers[3].mlp.experts, cfg.layers[3].mlp.top) == (56, 9, 4)
    assert cfg.layers[2].mlp is None
    cfg_b = arch.parse(pc.PS_B)
    assert cfg_b.loop is None and cfg_b.logit_softcap is None
    raw = copy.deepcopy(pc.PS_B)
    del raw["embedding"]
    assert arch.parse(raw).bigram is None and "bigram" not in DecoderModel.expected_tensors(spec_of(raw))
    with pytest.raises(ConfigError):
        arch.build_spec(cfg, window=8)


def test_layers_of_a_loop_run_in_order_with_what_joins_the_stream():
    calls = spec_of(pc.PS_A).schedule
    assert [(c.block, c.cache) for c in calls] == [
        ("l0", "l0"), ("l1", "l1"), ("l2", "l2"), ("l1", "l1.pass1"), ("l2", "l2.pass1"), ("l3", "l3")]
    assert [c.joins for c in calls] == [None, StreamInput(False, "loop.step", 0), None,
                                        StreamInput(True, "loop.step", 1), None, None]
    calls = spec_of(pc.PS_C).schedule
    assert [(c.block, c.joins and (c.joins.embedding, c.joins.row)) for c in calls] == [
        ("l0", (False, 0)), ("l0", (True, 1)), ("l0", (True, 2)), ("l1", None)]
    assert len({c.cache for c in calls}) == 4
    calls = spec_of(pc.PS_D).schedule
    assert [(c.block, c.joins and (c.joins.embedding, c.joins.row)) for c in calls] == [("l0", None), ("l1", (False, 0)), ("l2", None)]
    assert all(c.joins is None for c in spec_of(pc.PS_B).schedule)


def test_expected_tensors_and_cache_needs():
    names = DecoderModel.expected_tensors(spec_of(pc.PS_A))
    want = {"embed": (193, 48), "bigram": (102, 48), "loop.step": (2, 48), "head": (193, 48), "final.norm": (48,),
            "l0.norm1": (48,), "l0.mix.q": (72, 48), "l0.mix.dkv": (32, 48), "l0.mix.dkv.norm": (24,),
            "l0.mix.uk": (48, 24), "l0.mix.uv": (60, 24), "l0.mix.g": (60, 48), "l0.mix.o": (48, 60),
            "l0.mlp.router": (6, 48), "l0.mlp.e5.up": (40, 48), "l0.mlp.e5.down": (48, 40)}
    for name, shape in want.items():
        assert names[name].shape == shape, name
    for absent in ("l0.norm2", "l0.mix.sink", "l0.mlp.e6.up", "l0.mlp.e0.gate", "l0.mlp.correction", "l2.mlp.router", "l0.mix.dq"):
        assert absent not in names
    assert "loop.step" not in DecoderModel.expected_tensors(spec_of(pc.PS_B))
    needs = cpu_model(pc.PS_A).cache_needs()
    assert needs["embedding"] == StateNeed((1,), "int32")
    assert needs["l0"] == KVPagesNeed(1, 32, 9, 24, values_in_keys=True)
    assert needs["l1"] == needs["l1.pass1"] == KVPagesNeed(1, 52, 40, 40, values_in_keys=True)
    assert set(needs) == {"embedding", "l0", "l1", "l2", "l1.pass1", "l2.pass1", "l3"}
    assert cpu_model(pc.PS_C).graph_safe()


def _broken(path, value):
    raw = copy.deepcopy(pc.PS_A)
    at = raw
    for key in path[:-1]:
        at = at[key]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return raw


@pytest.mark.parametrize("path,value", [
    (("width",), None), (("vocab",), 0), (("norm", "eps"), 0.0), (("norm",), None), (("layers",), []),
    (("embedding", "bigram", "buckets"), 0), (("embedding", "bigram", "mul_prev"), None),
    (("embedding", "bigram", "mul_cur"), 1.5),
    (("layers", 0, "type"), "attention"), (("layers", 0, "mixer", "heads"), 0), (("layers", 0, "mixer", "kv_rank"), None),
    (("layers", 0, "mixer", "mask"), None), (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mixer", "scale"), "x"),
    (("layers", 0, "mixer", "rot"), None), (("layers", 0, "mixer", "rot", "dims"), 7), (("layers", 0, "mixer", "rot", "dims"), 10),
    (("layers", 0, "mixer", "rot", "base"), 0.0), (("layers", 0, "mlp", "kind"), "dense"),
    (("layers", 0, "mlp", "router", "top"), 7), (("layers", 0, "mlp", "expert"), None),
    (("loop", "stop"), 5), (("loop", "start"), 3), (("loop", "start"), -1), (("loop", "times"), 0), (("logit_softcap",), -2.0),
])
def test_refusals(path, value):
    with pytest.raises(ConfigError):
        architecture_of(pc.PS_A).parse(_broken(path, value))


def test_what_joins_the_stream_is_checked_by_the_model_spec():
    s = spec_of(pc.PS_A)
    make = lambda **kw: ModelSpec(**{**{f: getattr(s, f) for f in ("embedding", "blocks", "schedule", "final_norm",
                                                                    "final_norm_name", "head", "stream_tables")}, **kw})
    make()
    with pytest.raises(ValueError):
        make(schedule=(LayerCall("l0", "l0", StreamInput(table="loop.step", row=2)),))
    with pytest.raises(ValueError):
        make(schedule=(LayerCall("l0", "l0", StreamInput(table="other")),))
    with pytest.raises(ValueError):
        make(schedule=(LayerCall("l0", "embedding"),))
    with pytest.raises(ValueError):
        make(streams=2)


def test_sum_of_branches_in_front_of_a_norm_that_does_not_take_it():
    """Terms, rows and vector are added to the stream where the next norm does not do so in its own kernel, and
    handed on where it does; a branch of another kind stays pending and the rest joins the stream."""
    gen = torch.Generator().manual_seed(1)
    model = cpu_model(pc.PS_A)
    model.stream_tables["loop.step"] = torch.randn(2, 48, generator=gen)
    vec = model.stream_tables["loop.step"][1]
    x, a, emb = (torch.randn(5, 48, generator=gen) for _ in range(3))
    parts = torch.randn(3, 5, 48, generator=gen)
    joins = StreamInput(True, "loop.step", 1)
    takes, plain_norm = SimpleNamespace(TAKES_SUM=True), SimpleNamespace()
    resid = x.clone()
    got = model._join(resid, SumBranch((a, parts)), joins, emb, takes)
    assert torch.equal(resid, x) and got.terms == (a, parts) and got.extra is emb and torch.equal(got.vector, vec)
    assert model._join(resid, SumBranch((a, parts)), joins, emb, plain_norm) is None
    assert torch.allclose(resid, x + a + parts.sum(0) + emb + vec, atol=1e-5)
    resid = x.clone()
    assert model._join(resid, a, joins, emb, plain_norm) is None and torch.allclose(resid, x + a + emb + vec, atol=1e-5)
    resid, other = x.clone(), object()
    assert model._join(resid, other, joins, emb, takes) is other and torch.allclose(resid, x + emb + vec, atol=1e-5)
    assert model._join(resid, a, None, None, plain_norm) is a
    resid = x.clone()
    got = model._join(resid, None, StreamInput(False, "loop.step", 1), None, takes)
    assert got.terms == () and got.extra is None and torch.equal(got.vector, vec)


def _random_model(tag):
    from tokamak_b200.weights.random_init import random_tensors
    raw, init, _ = pc.ALL[tag]
    w = random_tensors(DecoderModel.expected_tensors(spec_of(raw)), dtype=torch.float32, **init)
    return raw, {k: v.double() for k, v in pc.sharpen(w, init["seed"], init["std"]).items()}


def test_random_folder_round_trip(tmp_path):
    folder = pc.write_folder(tmp_path / "m", "SB", "bfloat16")
    cfg, w = plain.load_folder(folder)
    assert cfg["architecture"] == "Puresun" and set(w) == set(DecoderModel.expected_tensors(spec_of(pc.PS_B)))
    logits = plain.forward(cfg, w, [1, 2, 3, 4, 5])
    assert logits.shape == (5, 157) and torch.isfinite(logits).all()


def test_plain_implementation_is_causal_and_its_pieces_agree():
    """A prefix's logits do not depend on what follows; pair rows follow the hash also where products leave 32
    bits; the rotation keeps lengths and depends on distance only; a window of one sees itself; the latent form of
    the scores is the product of full keys; router weights sum to one; rounding changes little."""
    raw, w = _random_model("SA")
    toks = [int(t) for t in torch.randint(0, 193, (60,), generator=torch.Generator().manual_seed(4))]
    full = plain.forward(raw, w, toks)
    assert (plain.forward(raw, w, toks[:31]) - full[:31]).abs().max() < 1e-9
    assert plain.bigram_rows([3, 5, 5], 101, 7, 13) == [101, (21 + 65) % 101, (35 + 65) % 101]
    assert plain.bigram_rows([156, 155], 4099, 7368787, 15485863)[1] == (156 * 7368787 + 155 * 15485863) % 4099
    assert 155 * 15485863 > 2 ** 31
    gen = torch.Generator().manual_seed(0)
    q, k = torch.randn(9, 2, 6, generator=gen, dtype=torch.float64), torch.randn(9, 2, 6, generator=gen, dtype=torch.float64)
    pos = torch.arange(9)
    a, b = plain.rotate_halves(q, pos, 4, 100.0), plain.rotate_halves(k, pos, 4, 100.0)
    assert (a.norm(dim=-1) - q.norm(dim=-1)).abs().max() < 1e-12 and torch.equal(a[..., 4:], q[..., 4:])
    a5, b5 = plain.rotate_halves(q, pos + 5, 4, 100.0), plain.rotate_halves(k, pos + 5, 4, 100.0)
    assert ((a[7] * b[3]).sum() - (a5[7] * b5[3]).sum()).abs() < 1e-12
    assert torch.equal(plain.window_mask(4, 1), torch.eye(4, dtype=torch.bool)) and plain.window_mask(6, 3)[5].tolist() == [
        False, False, False, True, True, True]
    # the attention written with full keys and values instead of latent queries
    m, eps = raw["layers"][1]["mixer"], 1e-5
    mw = plain.layer_weights(w, "l1.mix.")
    h = torch.randn(50, 48, generator=gen, dtype=torch.float64)
    H, d, dr, dv, r = (m[x] for x in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    down = h @ mw["dkv"].T
    c = plain.rms_norm(down[:, :r], mw["dkv.norm"], eps)
    kk = (c @ mw["uk"].T).view(50, H, d)
    vv = (c @ mw["uv"].T).view(50, H, dv)
    p50 = torch.arange(50)
    kr = plain.rotate_halves(down[:, None, r:], p50, dr, m["rot"]["base"]).expand(50, H, dr)
    qq = (h @ mw["q"].T).view(50, H, d + dr)
    qr = plain.rotate_halves(qq[..., d:], p50, dr, m["rot"]["base"])
    s = torch.einsum("ihd,jhd->hij", torch.cat([qq[..., :d], qr], -1), torch.cat([kk, kr], -1)) * m["scale"]
    s = s.masked_fill(~plain.window_mask(50, m["mask"]["size"]), float("-inf"))
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), vv).reshape(50, H * dv)
    want = (o * torch.sigmoid(h @ mw["g"].T)) @ mw["o"].T
    assert (plain.latent_attention(h, mw, m, eps, p50) - want).abs().max() < 1e-9
    idx, wt = plain.route(h, torch.randn(6, 48, generator=gen, dtype=torch.float64), 2)
    assert torch.allclose(wt.sum(-1), torch.ones(50, dtype=torch.float64)) and (wt[:, 0] >= wt[:, 1]).all()
    margins = []
    plain.forward(raw, w, toks, margins_out=margins)
    safe = torch.stack(margins).min(0).values.cummin(0).values > 0.05
    rounded = plain.forward(raw, w, toks, ROUND=plain.bf16_round)
    assert len(margins) == 4 and safe[0] and 0 < (rounded - full)[safe].abs().mean() < 0.1 * full.std()


def _lost_previous_token(monkeypatch):
    monkeypatch.setattr(plain, "bigram_rows", lambda toks, b, p, c, f=plain.bigram_rows: [
        b if i == 20 else r for i, r in enumerate(f(toks, b, p, c))])


def _window_off_by_one(monkeypatch):
    monkeypatch.setattr(plain, "window_mask", lambda T, size, f=plain.window_mask: f(T, size + 1))


def _window_one_short(monkeypatch):
    monkeypatch.setattr(plain, "window_mask", lambda T, size, f=plain.window_mask: f(T, max(1, size - 1)))


def _no_rotation(monkeypatch):
    monkeypatch.setattr(plain, "rotate_halves", lambda x, pos, dims, base: x)


def _softmax_over_all_experts(monkeypatch):
    def route(h, router, top):
        z = torch.softmax(h @ router.T, -1)
        vals, idx = torch.topk(z, top, dim=-1)
        return idx, vals
    monkeypatch.setattr(plain, "route", route)


def _pass_vector_of_the_first_pass_twice(monkeypatch):
    monkeypatch.setattr(plain, "run_order", lambda cfg, f=plain.run_order: [
        (i, 0 if p is not None else None) for i, p in f(cfg)])


@pytest.mark.parametrize("fault", [_lost_previous_token, _window_off_by_one, _window_one_short, _no_rotation,
                                   _softmax_over_all_experts, _pass_vector_of_the_first_pass_twice])
def test_mistakes_planted_in_the_oracle_show_in_the_logits(monkeypatch, fault):
    """The tests' weights are such that each of these faults moves some row by far more than the float32 tolerances
    and by more than the bfloat16 ones."""
    raw, w = _random_model("SA")
    toks = [int(t) for t in torch.randint(0, 193, (80,), generator=torch.Generator().manual_seed(5))]
    good = plain.forward(raw, w, toks)
    fault(monkeypatch)
    bad = plain.forward(raw, w, toks)
    rel = (bad - good).abs().amax(-1) / good.std(dim=-1)
    assert rel.max() > 0.3, rel.max()
