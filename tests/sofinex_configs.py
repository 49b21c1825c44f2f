"""Tiny Sofinex configurations for the tests.  They differ in every size and option: widths (also ones that are no
multiple of 8 or of 4), vocabularies, loops (none, from the first layer, in the middle, up to the last layer, one pass,
three), both mixers with all feed-forwards and without one, head counts, query/key and value sizes (equal, either one
larger, sizes that the tiled kernels take as they are, that are filled up to such a size, and beyond), whole and
partial rotation with and without scaling, windows of 1 token, inside a page, of several pages and longer than any
sequence, convolutions of 1 to 6 taps, ranks that are no multiple of 8, key heads shared by several value heads,
routers with and without identity experts, groups and a shared expert (smaller than an expert, equal, larger and no
multiple of it), inner sizes that the grouped products take and others, the cache's page size."""

from __future__ import annotations


def _wave(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def _yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def _att(heads, kv, dim, vdim, scale, window, dims, base, scaling):
    rot = {"base": base, "dims": dims}
    if scaling is not None:
        rot["scaling"] = scaling
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}, "rot": rot}


def _delta(heads, kv, dim, vdim, conv, decay_rank, gate_rank):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank,
            "gate_rank": gate_rank}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, identity, top, count, keep, shared):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top,
                                                            "groups": {"count": count, "keep": keep}}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def _diff_layer(att, diff, mlp):
    return {"type": "attention", "mixer": dict(att, diff=diff), "mlp": mlp}


def _pair_layer(left, right, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


SX_A = {
    "architecture": "Sofinex", "vocab": 173, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 0.8},
    "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        _diff_layer(_att(3, 1, 10, 14, 0.3, 9, 6, 500.0, _wave(3.0, 1.0, 4.0, 60)), 0.4, _moe(40, 6, 2, 3, 4, 2, 24)),
        _pair_layer(_att(4, 2, 12, 20, 0.25, 17, 8, 1000.0, _yarn(4.0, 40, 8.0, 1.0)), _delta(4, 2, 12, 10, 3, 5, 11),
                    _dense(72)),
        _diff_layer(_att(2, 2, 16, 8, 0.35, 1, 16, 10000.0, None), 0.2, None),
        _pair_layer(_att(3, 3, 18, 6, 0.2, 300, 18, 50000.0, None), _delta(3, 1, 7, 9, 1, 8, 3), None),
    ],
}
SX_B = {
    "architecture": "Sofinex", "vocab": 149, "width": 54, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.7},
    "layers": [
        _pair_layer(_att(2, 1, 9, 11, 0.3, 33, 4, 300.0, _yarn(8.0, 64, 32.0, 1.0)), _delta(2, 2, 20, 26, 6, 13, 20),
                    _moe(30, 5, 1, 2, 3, 2, 70)),
        _diff_layer(_att(6, 3, 7, 5, 0.4, 40, 2, 100.0, _wave(8.0, 0.5, 2.0, 100)), 0.6, _dense(50)),
    ],
}
# sizes that the products' own kernels and the tiled attention take (filled up), three passes from the first layer on
SX_C = {
    "architecture": "Sofinex", "vocab": 320, "width": 128, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.3},
    "loop": {"start": 0, "stop": 2, "times": 3},
    "layers": [
        _pair_layer(_att(8, 2, 48, 32, 0.15, 33, 32, 20000.0, _yarn(2.0, 128, 16.0, 2.0)), _delta(4, 2, 32, 64, 4, 16, 8),
                    _dense(256)),
        _diff_layer(_att(4, 1, 32, 64, 0.18, 80, 16, 5000.0, _wave(4.0, 1.0, 8.0, 256)), 0.3, _moe(64, 8, 8, 4, 4, 3, 128)),
        _diff_layer(_att(4, 2, 40, 72, 0.16, 48, 40, 1e6, _wave(16.0, 1.0, 1.5, 64)), 0.8, _moe(40, 7, 0, 2, 1, 1, None)),
    ],
}
# head sizes of 128, a single pass over a span that ends with the model, long ranks, one group
SX_D = {
    "architecture": "Sofinex", "vocab": 210, "width": 192, "norm": {"eps": 1e-5}, "embedding": {"scale": 0.9},
    "loop": {"start": 1, "stop": 3, "times": 1},
    "layers": [
        _diff_layer(_att(2, 1, 64, 128, 0.1, 20, 32, 10000.0, _wave(2.0, 1.0, 4.0, 100)), 0.5, _dense(384)),
        _pair_layer(_att(4, 1, 128, 96, 0.06, 100, 128, 150000.0, _yarn(4.0, 256, 32.0, 1.0)), _delta(3, 3, 64, 48, 2, 40, 72),
                    _moe(128, 10, 6, 5, 4, 2, 200)),
        _pair_layer(_att(2, 2, 70, 130, 0.1, 16, 60, 3000.0, None), _delta(2, 1, 136, 24, 5, 26, 18), _dense(100)),
    ],
}
# (configuration, how the random weights are drawn, page size)
ALL = {
    "XA": (SX_A, {"seed": 61, "std": 0.1, "norm_std": 0.1}, 16),
    "XB": (SX_B, {"seed": 62, "std": 0.1, "norm_std": 0.1}, 8),
    "XC": (SX_C, {"seed": 63, "std": 0.06, "norm_std": 0.1}, 32),
    "XD": (SX_D, {"seed": 64, "std": 0.06, "norm_std": 0.1}, 16),
}


def sharpen(tensors: dict, seed: int, std: float) -> dict:
    """Redraw what random draws leave without effect, so that every mechanism matters: routers that spread the
    scores and corrections of the scores' size, queries that tell keys apart (a window's edge shows), decays that keep
    a state alive for tens of tokens and differ from channel to channel, map weights near their middle."""
    import torch
    gen = torch.Generator().manual_seed(seed + 1000)
    for name in sorted(tensors):
        t, last = tensors[name], name.rsplit(".", 1)[-1]
        draw = torch.randn(t.shape, generator=gen)
        factor = {"router": 6.0, "q": 6.0, "g2": 4.0, "a2": 4.0, "b": 4.0, "sg": 4.0, "o": 3.0, "down": 3.0}.get(last)
        if name == "embed":
            new = draw
        elif last == "dt_bias":
            new = draw - 2.5
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            new = 0.6 * draw / t.shape[0] ** 0.25
        elif last == "correction":
            new = 0.1 * draw
        elif last == "norm1" or last == "norm2":
            new = 0.2 * draw
        elif last == "sink":
            new = 1.0 + draw
        elif factor is not None:
            new = factor * std * draw
        else:
            continue
        tensors[name] = new.to(t.dtype)
    return tensors


def write_folder(folder, tag: str, dtype: str):
    """A model folder of configuration ``tag``: seeded random weights, sharpened (:func:`sharpen`)."""
    from safetensors.torch import load_file, save_file

    from tokamak_b200.weights import write_random_model

    raw, init, _ = ALL[tag]
    write_random_model(folder, raw, dtype=dtype, **init)
    path = str(folder) + "/model.safetensors"
    tensors = sharpen(load_file(path), init["seed"], init["std"])
    save_file({k: v.contiguous() for k, v in tensors.items()}, path)
    return folder
