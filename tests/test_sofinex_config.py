"""The Sofinex design without a GPU: the reader of config.json and its refusals, the tensors it expects, the
order in which looped layers run and the caches they get, rotation frequencies, and the plain implementation's own
consistency and its sensitivity to planted mistakes."""

from __future__ import annotations

import copy
import math

import pytest
import torch

import sofinex_configs as sc
from plain import sofinex_plain as plain
from tokamak_b200.cache.manager import KVPagesNeed, StateNeed
from tokamak_b200.config.model_config import ConfigError
from tokamak_b200.config.registry import architecture_of, supported_architectures
from tokamak_b200.models.decoder import DecoderModel
from tokamak_b200.parts.base import Runtime
from tokamak_b200.parts.position import RopeHalvesSpec, WaveScaling, YarnScaling, scaled_frequencies


def spec_of(raw, shapes=None):
    arch = architecture_of(raw)
    return arch.build_spec(arch.parse(raw, tensor_shapes=shapes))


def cpu_model(raw, dtype=torch.float32):
    spec = spec_of(raw)
    names = DecoderModel.expected_tensors(spec)
    return DecoderModel(spec, {k: torch.zeros(r.shape, dtype=dtype if r.role == "matrix" else torch.float32)
                               for k, r in names.items()}, Runtime(device=torch.device("cpu"), dtype=dtype))


def test_registered_and_parsed():
    assert "Sofinex" in supported_architectures()
    arch = architecture_of(sc.SX_A)
    cfg = arch.parse(sc.SX_A)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.embedding_scale, cfg.loop) == (173, 48, 1e-5, 0.8, (1, 3, 2))
    m = cfg.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.window, m.diff) == (3, 1, 10, 14, 0.3, 9, 0.4)
    assert m.position == RopeHalvesSpec(6, 500.0, scaling=WaveScaling(3.0, 60.0, 1.0, 4.0))
    l, r = cfg.layers[1].mixer.left, cfg.layers[1].mixer.right
    assert l.position == RopeHalvesSpec(8, 1000.0, scaling=YarnScaling(4.0, 40.0, 8.0, 1.0)) and l.diff is None
    assert (r.heads, r.kv_heads, r.dim, r.vdim, r.conv, r.decay_rank, r.gate_rank) == (4, 2, 12, 10, 3, 5, 11)
    f = cfg.layers[0].mlp
    assert (f.ff, f.experts, f.identity, f.top, f.groups, f.keep, f.shared_ff) == (40, 6, 2, 3, 4, 2, 24)
    assert cfg.layers[1].mlp.ff == 72 and cfg.layers[2].mlp is None
    assert arch.parse(sc.SX_B).loop == (0, 0, 1)
    shapes = {"l1.mix.right.a1": (9, 48), "l1.mix.right.g1": (2, 48)}
    r = arch.parse(sc.SX_A, tensor_shapes=shapes).layers[1].mixer.right
    assert (r.decay_rank, r.gate_rank) == (9, 2)
    with pytest.raises(ConfigError):
        arch.build_spec(cfg, window=8)


def test_layers_of_a_loop_run_in_order_with_caches_of_their_own():
    calls = lambda raw: [(c.block, c.cache) for c in spec_of(raw).schedule]
    assert calls(sc.SX_A) == [("l0", "l0"), ("l1", "l1"), ("l2", "l2"), ("l1", "l1.pass1"), ("l2", "l2.pass1"), ("l3", "l3")]
    assert calls(sc.SX_B) == [("l0", "l0"), ("l1", "l1")]
    assert calls(sc.SX_C) == [("l0", "l0"), ("l1", "l1"), ("l0", "l0.pass1"), ("l1", "l1.pass1"), ("l0", "l0.pass2"),
                              ("l1", "l1.pass2"), ("l2", "l2")]
    assert calls(sc.SX_D) == [("l0", "l0"), ("l1", "l1"), ("l2", "l2")]
    for raw in (sc.SX_A, sc.SX_B, sc.SX_C, sc.SX_D):
        n, loop = len(raw["layers"]), raw.get("loop") or {"start": 0, "stop": 0, "times": 1}
        assert [int(b[1:]) for b, _ in calls(raw)] == plain.run_order(raw)
        assert len(calls(raw)) == n + (loop["stop"] - loop["start"]) * (loop["times"] - 1)


def test_expected_tensors_and_cache_needs():
    names = DecoderModel.expected_tensors(spec_of(sc.SX_A))
    want = {"embed": (173, 48), "head": (173, 48), "final.norm": (48,), "l0.norm1": (48,), "l0.norm2": (48,),
            "l0.mix.q": (60, 48), "l0.mix.k": (20, 48), "l0.mix.v": (14, 48), "l0.mix.lq1": (10,), "l0.mix.lk2": (10,),
            "l0.mix.o": (48, 42), "l0.mlp.router": (8, 48), "l0.mlp.correction": (8,), "l0.mlp.e5.gate": (40, 48),
            "l0.mlp.e5.down": (48, 40), "l0.mlp.shared.up": (24, 48), "l0.mlp.shared.sg": (1, 48),
            "l1.mix.left.q": (48, 48), "l1.mix.left.v": (40, 48), "l1.mix.left.sink": (4,), "l1.mix.left.o": (48, 80),
            "l1.mix.left.out": (48,), "l1.mix.right.q": (24, 48), "l1.mix.right.v": (40, 48), "l1.mix.right.v.conv": (40, 3),
            "l1.mix.right.b": (4, 48), "l1.mix.right.A_log": (4,), "l1.mix.right.a1": (5, 48), "l1.mix.right.a2": (48, 5),
            "l1.mix.right.dt_bias": (48,), "l1.mix.right.g1": (11, 48), "l1.mix.right.g2": (40, 11),
            "l1.mix.right.norm": (10,), "l1.mix.right.o": (48, 40), "l1.mix.right.out": (48,), "l1.mlp.up": (72, 48)}
    for name, shape in want.items():
        assert names[name].shape == shape, name
    for absent in ("l0.mlp.e6.gate", "l2.norm2", "l3.norm2", "l1.mix.right.a", "l1.mix.right.g", "l1.mlp.gate", "l0.mix.sink"):
        assert absent not in names
    assert "l2.mlp.shared.up" not in DecoderModel.expected_tensors(spec_of(sc.SX_C))
    needs = cpu_model(sc.SX_A).cache_needs()
    assert needs["l0"] == KVPagesNeed(1, 20, 9, 14)                 # one row holds both maps' keys
    assert needs["l1/left"] == needs["l1.pass1/left"] == KVPagesNeed(2, 12, 17, 20)
    assert needs["l1/right"] == StateNeed((4 * 12 * 10 + 2 * (2 * 24 + 40),), "float32")
    assert set(needs) == {"l0", "l1/left", "l1/right", "l2", "l1.pass1/left", "l1.pass1/right", "l2.pass1", "l3/left", "l3/right"}
    # in bfloat16 rows get a size of the tiled attention kernels, where there is one
    needs = cpu_model(sc.SX_D, torch.bfloat16).cache_needs()
    assert needs["l0"] == KVPagesNeed(1, 128, 20) and needs["l1/left"] == KVPagesNeed(1, 128, 100)
    assert needs["l2/left"] == KVPagesNeed(2, 70, 16, 130)
    assert cpu_model(sc.SX_C, torch.bfloat16).cache_needs()["l0/left"] == KVPagesNeed(2, 64, 33)
    assert cpu_model(sc.SX_C).graph_safe()


def _broken(path, value):
    raw = copy.deepcopy(sc.SX_A)
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
    (("embedding", "scale"), "x"), (("layers", 0, "type"), "delta"), (("layers", 0, "mixer", "heads"), 0),
    (("layers", 0, "mixer", "diff"), None), (("layers", 0, "mixer", "mask"), None), (("layers", 0, "mixer", "mask", "size"), 0),
    (("layers", 0, "mixer", "scale"), None), (("layers", 0, "mixer", "rot", "dims"), 5), (("layers", 0, "mixer", "rot", "dims"), 12),
    (("layers", 0, "mixer", "rot", "base"), 0.0), (("layers", 0, "mixer", "rot", "scaling", "low"), None),
    (("layers", 0, "mixer", "rot", "scaling", "high"), 0.5), (("layers", 1, "mixer", "left", "rot", "scaling", "fast"), None),
    (("layers", 1, "mixer", "left", "rot", "base"), 1.0), (("layers", 1, "mixer", "left", "kv_heads"), 3),
    (("layers", 1, "mixer", "right", "kv_heads"), 3), (("layers", 1, "mixer", "right", "conv"), 0),
    (("layers", 1, "mixer", "right"), None), (("layers", 0, "mlp", "kind"), "gated"), (("layers", 0, "mlp", "kind"), None),
    (("layers", 0, "mlp", "router", "top"), 5), (("layers", 0, "mlp", "router", "groups", "count"), 3),
    (("layers", 0, "mlp", "router", "groups", "keep"), 5), (("layers", 0, "mlp", "router", "identity"), -1),
    (("layers", 0, "mlp", "expert"), None), (("layers", 0, "mlp", "shared"), {}), (("layers", 1, "mlp", "ff"), 1.5),
    (("loop", "stop"), 5), (("loop", "start"), 4), (("loop", "start"), -1), (("loop", "times"), 0),
])
def test_refusals(path, value):
    with pytest.raises(ConfigError):
        architecture_of(sc.SX_A).parse(_broken(path, value))


@pytest.mark.parametrize("dims,base,factor,low,high,original", [
    (64, 10000.0, 8.0, 1.0, 4.0, 512), (12, 500.0, 2.0, 0.5, 1.5, 40), (2, 100.0, 3.0, 1.0, 4.0, 4), (32, 1e6, 1.0, 1.0, 4.0, 64)])
def test_frequencies_stretched_by_wavelength(dims, base, factor, low, high, original):
    got, mag = scaled_frequencies(dims, base, WaveScaling(factor, original, low, high))
    want, _ = plain.banded_frequencies(dims, base, {"factor": factor, "low": low, "high": high, "original": original})
    assert mag == 1.0 and torch.allclose(got, want, rtol=1e-12, atol=0.0)
    plain_f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    wave = 2 * math.pi / plain_f
    keep, slow = wave < original / high, wave > original / low
    assert torch.equal(got[keep], plain_f[keep]) or torch.allclose(got[keep], plain_f[keep], rtol=1e-15)
    assert torch.allclose(got[slow], plain_f[slow] / factor, rtol=1e-15)
    assert ((got <= plain_f * (1 + 1e-15)) & (got >= plain_f / factor * (1 - 1e-15))).all()


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [
    (80, 10000.0, 5.0, 600, 24.0, 1.0), (8, 500.0, 2.0, 64, 8.0, 2.0), (4, 100.0, 16.0, 4096, 32.0, 1.0), (64, 1e6, 1.0, 100, 4.0, 4.0)])
def test_frequencies_stretched_by_pair_index(dims, base, factor, original, fast, slow):
    got, mag = scaled_frequencies(dims, base, YarnScaling(factor, original, fast, slow))
    want, wmag = plain.ramped_frequencies(dims, base, {"factor": factor, "original": original, "fast": fast, "slow": slow})
    assert mag == wmag == 0.1 * math.log(factor) + 1.0 and torch.allclose(got, want, rtol=1e-12, atol=0.0)


def _random_model(tag):
    from tokamak_b200.weights.random_init import random_tensors
    raw, init, _ = sc.ALL[tag]
    w = random_tensors(DecoderModel.expected_tensors(spec_of(raw)), dtype=torch.float32, **init)
    return raw, {k: v.double() for k, v in sc.sharpen(w, init["seed"], init["std"]).items()}


def test_random_folder_round_trip(tmp_path):
    folder = sc.write_folder(tmp_path / "m", "XB", "bfloat16")
    cfg, w = plain.load_folder(folder)
    from tokamak_b200.weights.loader import checkpoint_shapes
    assert cfg["architecture"] == "Sofinex"
    assert set(w) == set(DecoderModel.expected_tensors(spec_of(sc.SX_B, checkpoint_shapes(folder))))
    logits = plain.forward(cfg, w, [1, 2, 3, 4, 5])
    assert logits.shape == (5, 149) and torch.isfinite(logits).all()


def test_plain_implementation_is_causal_and_its_pieces_agree():
    """A prefix's logits do not depend on what follows; the rotation keeps lengths and depends on distance only; the
    recurrence continues where it stopped and with one decay for all channels is the plain delta rule; the two maps
    with equal queries and keys cancel but for their weights; a sink takes its share; router weights sum to one."""
    raw, w = _random_model("XA")
    toks = [int(t) for t in torch.randint(0, 173, (60,), generator=torch.Generator().manual_seed(4))]
    full = plain.forward(raw, w, toks)
    assert (plain.forward(raw, w, toks[:31]) - full[:31]).abs().max() < 1e-9
    gen = torch.Generator().manual_seed(0)
    rand = lambda *s: torch.randn(*s, generator=gen, dtype=torch.float64)
    q, k, v = rand(9, 2, 6), rand(9, 2, 6), rand(9, 2, 3)
    pos = torch.arange(9)
    f, _ = plain.banded_frequencies(4, 100.0, None)
    a, b = plain.rotate_halves(q, pos, f), plain.rotate_halves(k, pos, f)
    assert (a.norm(dim=-1) - q.norm(dim=-1)).abs().max() < 1e-12 and torch.equal(a[..., 4:], q[..., 4:])
    a5, b5 = plain.rotate_halves(q, pos + 5, f), plain.rotate_halves(k, pos + 5, f)
    assert ((a[7] * b[3]).sum() - (a5[7] * b5[3]).sum()).abs() < 1e-12
    beta, g = torch.rand(9, 2, generator=gen, dtype=torch.float64), torch.rand(9, 2, 6, generator=gen, dtype=torch.float64)
    o, S = plain.delta_recurrence(q, k, v, beta, g)
    o1, S1 = plain.delta_recurrence(q[:4], k[:4], v[:4], beta[:4], g[:4])
    o2, S2 = plain.delta_recurrence(q[4:], k[4:], v[4:], beta[4:], g[4:], S1)
    assert (torch.cat([o1, o2]) - o).abs().max() < 1e-12 and (S2 - S).abs().max() < 1e-12
    # one step written out
    S0 = rand(2, 6, 3)
    o1, S1 = plain.delta_recurrence(q[:1], k[:1], v[:1], beta[:1], g[:1], S0)
    D = torch.diag(g[0, 1]) @ S0[1]
    want = D + torch.outer(k[0, 1], beta[0, 1] * (v[0, 1] - D.T @ k[0, 1]))
    assert (S1[1] - want).abs().max() < 1e-12 and (o1[0, 1] - want.T @ q[0, 1]).abs().max() < 1e-12
    att = plain.attend(q, k, v, 0.3, 4)
    sunk = plain.attend(q, k, v, 0.3, 4, torch.tensor([-1e9, 50.0], dtype=torch.float64))
    assert (sunk[:, 0] - att[:, 0]).abs().max() < 1e-12 and sunk[:, 1].abs().max() < 1e-12
    one = plain.attend(q, k, v, 0.3, 1)
    assert (one - v).abs().max() < 1e-12
    m = dict(raw["layers"][0]["mixer"])
    mw = plain.layer_weights(w, "l0.mix.")
    for n, rows in (("q", 3), ("k", 1)):
        t = mw[n].view(rows, 2, 10, 48).clone()
        t[:, 1] = t[:, 0]
        mw[n] = t.view(-1, 48)
    h = rand(20, 48)
    mw["lq1"], mw["lq2"] = torch.zeros(10, dtype=torch.float64), torch.zeros(10, dtype=torch.float64)
    m["diff"] = 0.25                                    # the second map then weighs 0.25: 0.75 of one map is left
    assert abs(plain.map_weight(mw, 0.25) - 0.25) < 1e-12
    f, _ = plain.banded_frequencies(6, 500.0, m["rot"]["scaling"])
    qq = plain.rotate_halves((h @ mw["q"].T).view(20, 6, 10), torch.arange(20), f)[:, ::2]
    kk = plain.rotate_halves((h @ mw["k"].T).view(20, 2, 10), torch.arange(20), f)[:, ::2]
    a1 = plain.attend(qq, kk, (h @ mw["v"].T).view(20, 1, 14), m["scale"], 9)
    y = plain.unit_rms(0.75 * a1, 1e-5).reshape(20, 42) * 0.75 @ mw["o"].T
    assert (plain.differential_attention(h, mw, m, 1e-5, torch.arange(20)) - y).abs().max() < 1e-9
    fw = plain.layer_weights(w, "l0.mlp.")
    chosen, weights, _ = plain.route(h, fw, raw["layers"][0]["mlp"]["router"])
    assert torch.allclose(weights.sum(-1), torch.ones(20, dtype=torch.float64)) and int(chosen.max()) >= 6
    assert all(len({int(e) // 2 for e in row}) <= 2 for row in chosen)
    big = plain.channel_decay(torch.full((1, 4), 50.0, dtype=torch.float64), torch.zeros(2, dtype=torch.float64),
                              torch.zeros(4, dtype=torch.float64))
    assert torch.allclose(big, torch.full_like(big, math.exp(-50.0)))


def _window(by):
    def fault(monkeypatch):
        monkeypatch.setattr(plain, "window_mask", lambda T, size, f=plain.window_mask: f(T, max(1, size + by)))
    return fault


def _patched(name, make):
    def fault(monkeypatch):
        monkeypatch.setattr(plain, name, make(getattr(plain, name)))
    return fault


FAULTS = {
    "window one longer": _window(1),
    "window one shorter": _window(-1),
    "no sink": _patched("attend", lambda f: lambda q, k, v, s, win, sink=None: f(q, k, v, s, win)),
    "second map not subtracted": _patched("map_weight", lambda f: lambda w, diff: 0.0 * f(w, diff)),
    "initial weight left out": _patched("map_weight", lambda f: lambda w, diff: f(w, 0.0)),
    "no rotation": _patched("rotate_halves", lambda f: lambda x, p, fr, m=1.0: x),
    "rotation's size lost": _patched("rotate_halves", lambda f: lambda x, p, fr, m=1.0: f(x, p, fr)),
    "frequencies not stretched by wavelength": _patched("banded_frequencies", lambda f: lambda d, b, s: f(d, b, None)),
    "state lost at position 20": _patched("delta_recurrence", lambda f: lambda q, k, v, b, g, s=None: (
        torch.cat([f(q[:20], k[:20], v[:20], b[:20], g[:20])[0], f(q[20:], k[20:], v[20:], b[20:], g[20:])[0]]), None)),
    "one decay per head": _patched("channel_decay", lambda f: lambda a, al, dt: f(a, al, dt).mean(-1, keepdim=True).expand(
        -1, -1, dt.numel() // al.numel())),
    "decays of the next channel": _patched("channel_decay", lambda f: lambda a, al, dt: f(a, al, dt).roll(1, -1)),
    "convolution lost at position 20": _patched("short_conv", lambda f: lambda x, t: torch.cat([f(x[:20], t), f(x[20:], t)])),
    "tanh form of gelu": _patched("gelu_exact", lambda f: lambda z: 0.5 * z * (1 + torch.tanh(0.9 * z))),
    "groups ignored": _patched("route", lambda f: lambda h, w, r: f(h, w, dict(r, groups={"count": 1, "keep": 1}))),
    "correction left out": _patched("route", lambda f: lambda h, w, r: f(h, dict(w, correction=0 * w["correction"]), r)),
    "weights not divided by their sum": _patched("route", lambda f: lambda h, w, r: (
        f(h, w, r)[0], torch.softmax(h @ w["router"].T, -1).gather(1, f(h, w, r)[0]), None)),
    "norm's weight around one": _patched("offset_norm", lambda f: lambda x, w, eps: plain.unit_rms(x, eps) * w),
}


@pytest.mark.parametrize("name", list(FAULTS))
def test_mistakes_planted_in_the_oracle_show_in_the_logits(monkeypatch, name):
    """The tests' weights are such that each of these faults moves some row by far more than the float32 tolerances
    and, but for the two small ones, by more than the bfloat16 ones."""
    least = 0.1 if name in ("rotation's size lost", "tanh form of gelu") else 0.25
    raw, w = _random_model("XA")
    toks = [int(t) for t in torch.randint(0, 173, (80,), generator=torch.Generator().manual_seed(5))]
    good = plain.forward(raw, w, toks)
    FAULTS[name](monkeypatch)
    bad = plain.forward(raw, w, toks)
    rel = (bad - good).abs().amax(-1) / good.std(dim=-1)
    assert rel.max() > least, rel.max()
