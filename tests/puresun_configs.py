"""Tiny Puresun configurations for the tests.  They differ in every size and option: widths (also ones that are no
multiple of 8 or of 4), vocabularies, pair tables (few buckets, more buckets than pairs ever hit, multipliers
whose products leave 32 bits), loops (none, from the first layer, in the middle, up to the last layer, one pass,
three), layers without a feed-forward, head counts (1 to 18), query/key, value and latent sizes (latents in steps
of 16, which the tensor-core attention takes, and others), rotated parts turned whole, windows of 1 token,
inside a page, of several pages and longer than any sequence, numbers of experts and of chosen ones (1, some,
all), inner sizes that the grouped products take and others, capped and uncapped logits, the cache's page size."""

from __future__ import annotations


def _mixer(heads, dim, rot_dim, vdim, rank, scale, window, base=10000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
            "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim}}


def _moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _layer(mixer, mlp):
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def _bigram(buckets, mul_prev, mul_cur):
    return {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}


PS_A = {
    "architecture": "Puresun", "vocab": 193, "width": 48, "norm": {"eps": 1e-5}, "embedding": _bigram(101, 7, 13),
    "loop": {"start": 1, "stop": 3, "times": 2}, "logit_softcap": 12.0,
    "layers": [
        _layer(_mixer(3, 16, 8, 20, 24, 0.3, 9), _moe(40, 6, 2)),
        _layer(_mixer(2, 8, 12, 10, 40, 0.25, 40, base=500.0), _moe(24, 4, 1)),
        _layer(_mixer(5, 10, 4, 6, 18, 0.35, 1), None),
        _layer(_mixer(1, 32, 16, 48, 12, 0.2, 300, base=1e6), _moe(56, 9, 4)),
    ],
}
PS_B = {
    "architecture": "Puresun", "vocab": 157, "width": 54, "norm": {"eps": 1e-6}, "embedding": _bigram(4099, 7368787, 15485863),
    "layers": [
        _layer(_mixer(4, 8, 6, 40, 20, 0.4, 17), None),
        _layer(_mixer(6, 12, 10, 8, 30, 0.3, 64), _moe(30, 3, 3)),
    ],
}
# sizes that the products' own kernels and the tensor-core attention take, three passes from the first layer on
PS_C = {
    "architecture": "Puresun", "vocab": 320, "width": 128, "norm": {"eps": 1e-5}, "embedding": _bigram(257, 1, 19),
    "loop": {"start": 0, "stop": 1, "times": 3}, "logit_softcap": 20.0,
    "layers": [
        _layer(_mixer(4, 32, 32, 48, 64, 0.125, 33), _moe(64, 8, 2)),
        _layer(_mixer(8, 64, 16, 32, 128, 0.11, 80, base=50000.0), _moe(104, 12, 3)),
    ],
}
# head counts that fill no tile evenly, a single pass over a span that ends with the model
PS_D = {
    "architecture": "Puresun", "vocab": 222, "width": 192, "norm": {"eps": 1e-5}, "embedding": _bigram(29, 5, 3),
    "loop": {"start": 1, "stop": 3, "times": 1}, "logit_softcap": 25.0,
    "layers": [
        _layer(_mixer(18, 8, 16, 24, 80, 0.2, 20), _moe(72, 16, 1)),
        _layer(_mixer(7, 24, 16, 40, 48, 0.16, 100, base=2000.0), _moe(128, 5, 2)),
        _layer(_mixer(5, 16, 32, 16, 32, 0.22, 16), _moe(40, 10, 5)),
    ],
}
# (configuration, how the random weights are drawn, page size)
ALL = {
    "SA": (PS_A, {"seed": 51, "std": 0.1, "norm_std": 0.1}, 16),
    "SB": (PS_B, {"seed": 52, "std": 0.1, "norm_std": 0.1}, 8),
    "SC": (PS_C, {"seed": 53, "std": 0.06, "norm_std": 0.1}, 32),
    "SD": (PS_D, {"seed": 54, "std": 0.06, "norm_std": 0.1}, 16),
}


def sharpen(tensors: dict, seed: int, std: float) -> dict:
    """Redraw what random draws leave without effect, so that every mechanism matters: routers that spread the
    scores, queries that tell keys apart (a window's edge shows), gates that are not all half open, embedded rows
    and pair rows of a size that the first layers do not drown."""
    import torch
    gen = torch.Generator().manual_seed(seed + 1000)
    for name in sorted(tensors):
        t = tensors[name]
        factor = {"router": 8.0, "q": 6.0, "g": 4.0}.get(name.rsplit(".", 1)[-1])
        if name in ("embed", "bigram"):
            tensors[name] = torch.randn(t.shape, generator=gen).to(t.dtype)
        elif factor is not None:
            tensors[name] = (factor * std * torch.randn(t.shape, generator=gen)).to(t.dtype)
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
