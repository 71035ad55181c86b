"""The Pirozen design, plainly: whole sequences, one function per mechanism, 64-bit unless told otherwise, no cache and no
code shared with the package.  `forward(cfg, tensors, tokens)` returns the logits of every position (and, on request,
the residual stream after every layer run); `tensors` maps the stored names to torch tensors, `cfg` is config.json as a dict.

Notation: W x for a stored matrix W [out, in]; t, j positions of one sequence counted from 0; h the input of a sublayer.

    stream         x_t = E[token_t] =: x0_t
    layer          x <- x + (mixer(rms(x) w1) + ff(rms(x) w2)),  then with g = gelu_tanh(A x) * S[token, layer's part]:
                   x <- x + rms(B g) w3
    loop           layers start .. stop-1 run `times` times in a row, x <- W [x; x0] ahead of each of these passes
    attention      biased projections, q and k normed per head, pairs (i, i + dims/2) turned by stretched frequencies, causal
                   softmax over the last `size` positions, a head's output times the sigmoid of one number, biased W_o
    feed-forward   `top` of the experts and identities by softmax score + correction, out of the best groups; weights are
                   their scores over the scores' sum, times a factor; an expert is down(silu(gate h) * up h), an identity h;
                   plus one more expert for every token
    head           W rms(x) w
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def stretched(rot):
    """(frequencies, factor on cosines and sines) of a rotation of rot["dims"] dimensions."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    freqs = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not sc:
        return freqs, 1.0

    def dim_of(turns):
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), n - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, D]: pairs (i, i + dims/2) of the first `dims` dimensions turn by t f_i; the rest passes."""
    freqs, factor = stretched(rot)
    out, half = x.clone(), rot["dims"] // 2
    t = torch.arange(x.shape[0], dtype=torch.float64)
    for i, f in enumerate(freqs):
        c, s = (torch.cos(t * f) * factor).to(x.dtype)[:, None], (torch.sin(t * f) * factor).to(x.dtype)[:, None]
        out[..., i] = x[..., i] * c - x[..., i + half] * s
        out[..., i + half] = x[..., i + half] * c + x[..., i] * s
    return out


def windowed_softmax(q, k, v, scale, size):
    """q [H, T, D], k [H, T, D], v [H, T, V] (keys and values already one per query head)."""
    T = q.shape[1]
    t, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    visible = (j <= t) & (t - j < size)
    s = (q @ k.transpose(1, 2) * scale).masked_fill(~visible, float("-inf"))
    return torch.softmax(s, dim=-1) @ v


def attention(m, tensors, pre, h, eps, dt):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    W = lambda n: tensors[pre + n].to(dt)
    q = (h @ W("q").T + W("q.b")).reshape(T, H, D)
    k = (h @ W("k").T + W("k.b")).reshape(T, G, D)
    v = (h @ W("v").T + W("v.b")).reshape(T, G, V).permute(1, 0, 2).repeat_interleave(H // G, dim=0)
    q, k = rotate(rms(q, eps) * W("q.norm"), m["rot"]), rotate(rms(k, eps) * W("k.norm"), m["rot"])
    k = k.permute(1, 0, 2).repeat_interleave(H // G, dim=0)
    o = windowed_softmax(q.permute(1, 0, 2), k, v, m["scale"], m["mask"]["size"]).permute(1, 0, 2)      # [T, H, V]
    o = o * torch.sigmoid(h @ W("g").T)[:, :, None]
    return o.reshape(T, H * V) @ W("o").T + W("o.b")


def unit(tensors, pre, h, dt):
    W = lambda n: tensors[pre + n].to(dt)
    return (silu(h @ W("gate").T) * (h @ W("up").T)) @ W("down").T


def choose(s, correction, router):
    """The chosen outputs of one token: s and correction are lists of numbers, one per expert and identity."""
    n, top = len(s), router["top"]
    choice = [a + b for a, b in zip(s, correction)]
    if router.get("groups"):
        count, keep = router["groups"]["count"], router["groups"]["keep"]
        size = n // count
        best = [max(choice[g * size:(g + 1) * size]) for g in range(count)]
        kept = sorted(range(count), key=lambda g: (-best[g], g))[:keep]
        choice = [c if e // size in kept else float("-inf") for e, c in enumerate(choice)]
    return sorted(range(n), key=lambda e: (-choice[e], e))[:top]


def margin(s, correction, router):
    """How far the choice of one token is from another one: the smaller of the distances between the last chosen and the first
    left-out expert of the kept groups, and between the last kept and the first dropped group."""
    n = len(s)
    choice = [a + b for a, b in zip(s, correction)]
    out, kept = float("inf"), range(n)
    if router.get("groups"):
        count, keep = router["groups"]["count"], router["groups"]["keep"]
        size = n // count
        best = sorted(((max(choice[g * size:(g + 1) * size]), -g) for g in range(count)), reverse=True)
        if keep < count:
            out = best[keep - 1][0] - best[keep][0]
        groups = {-g for _, g in best[:keep]}
        kept = [e for e in range(n) if e // size in groups]
    ranked = sorted((choice[e] for e in kept), reverse=True)
    if router["top"] < len(ranked):
        out = min(out, ranked[router["top"] - 1] - ranked[router["top"]])
    return out


def feed_forward(mlp, tensors, pre, h, dt, margins_out=None):
    """`margins_out`: a list that receives every token's `margin` (where that is tiny, a lower precision may choose otherwise)."""
    W = lambda n: tensors[pre + n].to(dt)
    r = mlp["router"]
    real = r["experts"]
    s = torch.softmax(h @ W("router").T, dim=-1)
    corr = W("correction")
    if margins_out is not None:
        margins_out.append(torch.tensor([margin(s[t].tolist(), corr.tolist(), r) for t in range(h.shape[0])]))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = choose(s[t].tolist(), corr.tolist(), r)
        total = sum(s[t, e] for e in chosen) + 1e-20
        for e in chosen:
            y = unit(tensors, f"{pre}e{e}.", h[t:t + 1], dt)[0] if e < real else h[t]
            out[t] += s[t, e] / total * r["scale"] * y
    if mlp.get("shared"):
        out = out + unit(tensors, pre + "shared.", h, dt)
    return out


def token_input(tensors, i, dim, tokens, x, eps, dt):
    """The term that layer i adds from its part of the tokens' side rows."""
    W = lambda n: tensors[f"l{i}.side.{n}"].to(dt)
    e = tensors["side.embed"].to(dt)[torch.tensor(tokens, dtype=torch.long)][:, i * dim:(i + 1) * dim]
    return rms((gelu_tanh(x @ W("gate").T) * e) @ W("proj").T, eps) * W("norm")


def runs(cfg):
    """The layer runs of one forward pass, None standing for the step ahead of a pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    inner = [None] + list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inner * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, tensors, tokens, dt=torch.float64, layers_out=None, margins_out=None):
    eps = cfg["norm"]["eps"]
    norm = lambda x, name: rms(x, eps) * tensors[name].to(dt)
    x0 = tensors["embed"].to(dt)[torch.tensor(tokens, dtype=torch.long)]
    x = x0
    for i in runs(cfg):
        if i is None:
            x = torch.cat([x, x0], dim=-1) @ tensors["loop.in"].to(dt).T
            continue
        pre, layer = f"l{i}.", cfg["layers"][i]
        y = attention(layer["mixer"], tensors, pre + "mix.", norm(x, pre + "norm1"), eps, dt)
        if layer["mlp"] is not None:
            y = y + feed_forward(layer["mlp"], tensors, pre + "mlp.", norm(x, pre + "norm2"), dt, margins_out)
        x = x + y
        if cfg.get("token_side"):
            x = x + token_input(tensors, i, cfg["token_side"]["dim"], tokens, x, eps, dt)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ tensors["head"].to(dt).T
