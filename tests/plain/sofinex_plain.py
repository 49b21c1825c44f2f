"""A slow, plain implementation of the Sofinex design, one function per mechanism, written from the
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


# ---- norms and activations

def unit_rms(x, eps):
    """Divided by the root mean square of the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu_exact(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ---- rotation

def banded_frequencies(dims, base, sc):
    """Frequencies scaled by wavelength: short waves keep theirs, long ones are divided by the factor, a linear
    blend between (in the number of waves that fit into the original length)."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=DT), 1.0


def ramped_frequencies(dims, base, sc):
    """Frequencies scaled by pair index: a ramp between the pair that turns ``fast`` times over the original length
    and the one that turns ``slow`` times; cosine and sine grow with the logarithm of the factor."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return torch.tensor(freq, dtype=DT), 1.0

    def at(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return torch.tensor(out, dtype=DT), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x, positions, freq, magnitude=1.0):
    """x [T, H, d]: elements (i, i + n) of the first 2 n turn by position * freq[i], n = len(freq)."""
    n = len(freq)
    ang = positions.to(DT)[:, None] * freq[None, :]
    c, s = (torch.cos(ang) * magnitude)[:, None, :], (torch.sin(ang) * magnitude)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


# ---- attention

def window_mask(T, size):
    """[T, T] bool: query i sees key j with 0 <= i - j < size."""
    i = torch.arange(T)
    dist = i[:, None] - i[None, :]
    return (dist >= 0) & (dist < size)


def attend(q, k, v, scale, window, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: softmax over the window, query head h reads head h // (H / G);
    ``sink`` [H]: a number per head whose exponential joins the denominator."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    k, v = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~window_mask(T, window), -math.inf)
    if sink is not None:
        p = torch.softmax(torch.cat([s, sink[:, None, None].expand(H, T, 1)], dim=-1), dim=-1)[..., :-1]
    else:
        p = torch.softmax(s, dim=-1)
    return torch.einsum("hij,jhd->ihd", p, v)


def map_weight(w, diff):
    """The weight of the second map: one number per layer."""
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def differential_attention(h, w, m, eps, positions, ROUND=no_round):
    """Two attention maps per head over the same values; the second is subtracted."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freq, mag = banded_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = ROUND(h @ w["q"].T).view(T, H * 2, d)
    k = ROUND(h @ w["k"].T).view(T, G * 2, d)
    v = ROUND(h @ w["v"].T).view(T, G, dv)
    q, k = (ROUND(rotate_halves(t, positions, freq, mag)) for t in (q, k))
    q, k = q.view(T, H, 2, d), k.view(T, G, 2, d)
    a1, a2 = (ROUND(attend(q[:, :, i], k[:, :, i], v, m["scale"], m["mask"]["size"])) for i in (0, 1))
    o = unit_rms(a1 - map_weight(w, m["diff"]) * a2, eps) * (1.0 - m["diff"])
    return ROUND(ROUND(o.reshape(T, H * dv)) @ w["o"].T)


def sink_attention(h, w, m, eps, positions, ROUND=no_round):
    """q and k heads divided by their root mean square after the rotation, a sink per head."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freq, mag = ramped_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = ROUND(h @ w["q"].T).view(T, H, d)
    k = ROUND(h @ w["k"].T).view(T, G, d)
    v = ROUND(h @ w["v"].T).view(T, G, dv)
    q, k = (ROUND(unit_rms(rotate_halves(t, positions, freq, mag), eps)) for t in (q, k))
    a = ROUND(attend(q, k, v, m["scale"], m["mask"]["size"], w["sink"]))
    return ROUND(a.reshape(T, H * dv) @ w["o"].T)


# ---- the delta rule with a decay per key channel

def short_conv(x, taps):
    """x [T, C], taps [C, K]: causal, the last tap weighs the current row; silu follows."""
    T, K = x.shape[0], taps.shape[1]
    pad = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x])
    return silu(sum(pad[j:j + T] * taps[:, j] for j in range(K)))


def unit_vector(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def delta_recurrence(q, k, v, beta, g, state=None):
    """q, k [T, H, dk], v [T, H, dv], beta [T, H], g [T, H, dk]; returns (o [T, H, dv], the last state)."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=v.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def channel_decay(a, a_log, dt_bias):
    """a [T, H * dk], a_log [H], dt_bias [H * dk] -> decays [T, H, dk] in (0, 1]."""
    T, H = a.shape[0], a_log.shape[0]
    return torch.exp(-torch.exp(a_log)[None, :, None] * softplus(a + dt_bias).view(T, H, -1))


def delta_mixer(h, w, m, eps, ROUND=no_round):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(ROUND(h @ w[n].T), w[n + ".conv"]) for n in ("q", "k", "v"))
    q, k = unit_vector(q.view(T, G, dk)) * dk ** -0.5, unit_vector(k.view(T, G, dk))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(ROUND(h @ w["b"].T))
    g = channel_decay(ROUND(ROUND(h @ w["a1"].T) @ w["a2"].T), w["A_log"], w["dt_bias"])
    o, _ = delta_recurrence(q, k, v.view(T, H, dv), beta, g)
    gate = torch.sigmoid(ROUND(ROUND(h @ w["g1"].T) @ w["g2"].T))
    y = ROUND(unit_rms(o, eps) * w["norm"]).reshape(T, H * dv) * gate
    return ROUND(ROUND(y) @ w["o"].T)


def side_by_side(h, w, m, eps, positions, ROUND=no_round):
    """Half the sum of two mixers' outputs, each normed over the model's width."""
    left = sink_attention(h, layer_weights(w, "left."), m["left"], eps, positions, ROUND)
    right = delta_mixer(h, layer_weights(w, "right."), m["right"], eps, ROUND)
    return 0.5 * (unit_rms(left, eps) * w["left.out"] + unit_rms(right, eps) * w["right.out"])


# ---- feed-forwards

def dense_ff(h, w, ROUND=no_round):
    return ROUND(ROUND(gelu_exact(ROUND(h @ w["up"].T))) @ w["down"].T)


def gated_ff(x, gate, up, down, ROUND=no_round):
    return ROUND(ROUND(silu(ROUND(x @ gate.T)) * ROUND(x @ up.T)) @ down.T)


def choice_scores(h, router, correction):
    s = torch.softmax(h @ router.T, dim=-1)
    return s, s + correction


def route(h, w, r):
    """(chosen [T, top], weights [T, top], margins [T]): softmax scores over all outputs; the choice by score plus
    correction among the groups whose best choice score is largest; the chosen scores divided by their sum.
    A margin is by how much the closest of the two decisions was taken."""
    total = r["experts"] + r.get("identity", 0)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    count, keep, top = groups["count"], groups["keep"], r["top"]
    s, c = choice_scores(h, w["router"], w["correction"])
    T = h.shape[0]
    best = c.view(T, count, total // count).max(-1).values
    order = best.sort(-1, descending=True)
    margin = torch.full((T,), math.inf, dtype=h.dtype)
    if keep < count:
        margin = order.values[:, keep - 1] - order.values[:, keep]
    allowed = torch.zeros(T, count, dtype=torch.bool).scatter_(1, order.indices[:, :keep], True)
    allowed = allowed.repeat_interleave(total // count, dim=1)
    c = c.masked_fill(~allowed, -math.inf)
    ranked = c.sort(-1, descending=True)
    if top < keep * (total // count):
        margin = torch.minimum(margin, ranked.values[:, top - 1] - ranked.values[:, top])
    chosen = ranked.indices[:, :top]
    weights = s.gather(1, chosen)
    return chosen, weights / (weights.sum(-1, keepdim=True) + 1e-20), margin


def mixture(h, w, mlp, ROUND=no_round, margins_out=None):
    """Weighted sum of the chosen experts (the last ones hand the input on) plus the gated shared expert."""
    r = mlp["router"]
    chosen, weights, margin = route(h, w, r)
    if margins_out is not None:
        margins_out.append(margin)
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r.get("identity", 0)):
        t, k = torch.nonzero(chosen == e, as_tuple=True)
        if len(t) == 0:
            continue
        y = gated_ff(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], ROUND) if e < r["experts"] else h[t]
        out[t] += weights[t, k][:, None] * y
    if mlp.get("shared") is not None:
        gate = torch.sigmoid(ROUND(h @ w["shared.sg"].T))
        out = out + gate * gated_ff(h, w["shared.gate"], w["shared.up"], w["shared.down"], ROUND)
    return out


# ---- the model

def layer_weights(weights, prefix):
    return {k[len(prefix):]: t for k, t in weights.items() if k.startswith(prefix)}


def run_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def layer(x, cfg, lay, w, positions, ROUND=no_round, margins_out=None):
    eps = cfg["norm"]["eps"]
    h = ROUND(offset_norm(x, w["norm1"], eps))
    mix = layer_weights(w, "mix.")
    if lay["type"] == "parallel":
        x = x + side_by_side(h, mix, lay["mixer"], eps, positions, ROUND)
    else:
        x = x + differential_attention(h, mix, lay["mixer"], eps, positions, ROUND)
    if lay.get("mlp") is None:
        return x
    h = ROUND(offset_norm(x, w["norm2"], eps))
    mlp = layer_weights(w, "mlp.")
    if lay["mlp"]["kind"] == "dense":
        return x + dense_ff(h, mlp, ROUND)
    return x + mixture(h, mlp, lay["mlp"], ROUND, margins_out)


def forward(cfg, weights, tokens, ROUND=no_round, layers_out=None, margins_out=None):
    """Logits [T, vocab] of one sequence from position 0; ``weights`` maps names to float64 tensors.
    ``layers_out``: a list that receives the residual stream after every layer run;
    ``margins_out``: one that receives every router's margins."""
    positions = torch.arange(len(tokens))
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i in run_order(cfg):
        x = layer(x, cfg, cfg["layers"][i], layer_weights(weights, f"l{i}."), positions, ROUND, margins_out)
        if layers_out is not None:
            layers_out.append(x)
    return ROUND(offset_norm(x, weights["final.norm"], cfg["norm"]["eps"])) @ weights["head"].T


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
