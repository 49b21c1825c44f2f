"""A slow, plain implementation of the Puresun design, one function per mechanism, written from the
design's equations.  It shares no code with the package: tensors in, tensors out, a whole sequence at
a time, float64 unless the caller says otherwise.  ``ROUND`` (a function tensor -> tensor) rounds
where an engine of 16 bits rounds: the results of matrix products and the rows that feed them.

Notation: ``x`` rows are tokens ``[T, width]``; ``W`` matrices are ``[out, in]`` and applied as ``x @ W.T``.
"""

from __future__ import annotations

import math

import torch

DT = torch.float64


def no_round(t):
    return t


def bf16_round(t):
    return t.to(torch.bfloat16).to(t.dtype)


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token: a hash of (previous, current), the last row for the first token."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return rows[:len(tokens)]


def embedding(weights, tokens, bigram):
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    if bigram:
        rows = bigram_rows(tokens, bigram["buckets"], bigram["mul_prev"], bigram["mul_cur"])
        x = x + weights["bigram"][torch.tensor(rows)]
    return x


def rotate_halves(x, positions, dims, base):
    """x [T, H, d]: elements (i, i + dims / 2) of the first ``dims`` turn by position * base^(-2i / dims)."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=DT)
    ang = positions.to(DT)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def window_mask(T, size):
    """[T, T] bool: query i sees key j with 0 <= i - j < size."""
    i = torch.arange(T)
    dist = i[:, None] - i[None, :]
    return (dist >= 0) & (dist < size)


def latent_attention(h, w, m, eps, positions, ROUND=no_round):
    """Keys and values of every head are products of one normed latent per token; one rotated key part is
    shared by the heads; softmax over a sliding window; a sigmoid gate per channel."""
    T = h.shape[0]
    H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = ROUND(h @ w["q"].T).view(T, H, d + dr)
    down = ROUND(h @ w["dkv"].T)
    c = ROUND(rms_norm(down[:, :r], w["dkv.norm"], eps))
    k_rot = ROUND(rotate_halves(down[:, None, r:], positions, m["rot"]["dims"], m["rot"]["base"]))[:, 0]
    q_rot = ROUND(rotate_halves(q[..., d:], positions, m["rot"]["dims"], m["rot"]["base"]))
    # the scores in the latent space: q . (W_uk c) = (W_uk^T q) . c
    wuk, wuv = w["uk"].view(H, d, r), w["uv"].view(H, dv, r)
    q_lat = ROUND(torch.einsum("thd,hdr->thr", q[..., :d], wuk))
    s = (torch.einsum("ihr,jr->hij", q_lat, c) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    s = s.masked_fill(~window_mask(T, m["mask"]["size"]), -math.inf)
    p = torch.softmax(s, dim=-1)
    o = torch.einsum("htr,hdr->thd", ROUND(torch.einsum("hij,jr->hir", p, c)), wuv)
    y = ROUND(o).reshape(T, H * dv) * torch.sigmoid(ROUND(h @ w["g"].T))
    return ROUND(ROUND(y) @ w["o"].T)


def route(h, router, top):
    """(chosen experts [T, top], their weights [T, top]): the largest logits, softmax over the chosen only."""
    z = h @ router.T
    vals, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(vals, dim=-1)


def expert_ff(x, up, down, ROUND=no_round):
    a = torch.relu(ROUND(x @ up.T))
    return ROUND(ROUND(a * a) @ down.T)


def choice_margin(h, router, top):
    """[T] by how much the last chosen logit beats the first one that is not chosen."""
    z = (h @ router.T).sort(-1, descending=True).values
    return z[:, top - 1] - z[:, top] if top < z.shape[1] else torch.full((z.shape[0],), math.inf, dtype=z.dtype)


def mixture(h, w, mlp, ROUND=no_round, margins_out=None):
    """The weighted sum of the chosen experts' outputs."""
    idx, weight = route(h, w["router"], mlp["router"]["top"])
    if margins_out is not None:
        margins_out.append(choice_margin(h, w["router"], mlp["router"]["top"]))
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, k = torch.nonzero(idx == e, as_tuple=True)
        if len(t):
            out[t] += weight[t, k][:, None] * expert_ff(h[t], w[f"e{e}.up"], w[f"e{e}.down"], ROUND)
    return out


def layer_weights(weights, prefix):
    return {k[len(prefix):]: t for k, t in weights.items() if k.startswith(prefix)}


def run_order(cfg):
    """[(layer, pass or None)]: the pass of a looped layer is given for its span's first layer only."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def parallel_layer(x, cfg, lay, w, positions, ROUND=no_round, margins_out=None):
    """x + (mixer(h) + ff(h)) with one norm in front of both."""
    eps = cfg["norm"]["eps"]
    h = ROUND(rms_norm(x, w["norm1"], eps))
    y = latent_attention(h, layer_weights(w, "mix."), lay["mixer"], eps, positions, ROUND)
    if lay.get("mlp") is not None:
        y = y + mixture(h, layer_weights(w, "mlp."), lay["mlp"], ROUND, margins_out)
    return x + y


def forward(cfg, weights, tokens, ROUND=no_round, layers_out=None, margins_out=None):
    """Logits [T, vocab] of one sequence from position 0; ``weights`` maps names to float64 tensors.
    ``layers_out``: a list that receives the residual stream after every layer run;
    ``margins_out``: one that receives every router's margins."""
    positions = torch.arange(len(tokens))
    emb = embedding(weights, tokens, (cfg.get("embedding") or {}).get("bigram"))
    x = emb.clone()
    for i, p in run_order(cfg):
        if p is not None:
            if p > 0:
                x = x + emb
            x = x + weights["loop.step"][p]
        x = parallel_layer(x, cfg, cfg["layers"][i], layer_weights(weights, f"l{i}."), positions, ROUND, margins_out)
        if layers_out is not None:
            layers_out.append(x)
    logits = ROUND(rms_norm(x, weights["final.norm"], cfg["norm"]["eps"])) @ weights["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


def load_folder(folder):
    """``(config dictionary, name -> float64 tensor)`` of a model folder."""
    import json
    from pathlib import Path

    from safetensors.torch import load_file
    cfg = json.loads((Path(folder) / "config.json").read_text())
    return cfg, {k: v.to(DT) for k, v in load_file(str(Path(folder) / "model.safetensors")).items()}


def greedy_generate(cfg, weights, prompt, n_new):
    seq, out = list(prompt), []
    for _ in range(n_new):
        tok = int(forward(cfg, weights, seq)[-1].argmax())
        out.append(tok)
        seq.append(tok)
    return out
