"""The Sogenex design, plainly: whole sequences, one function per mechanism, 64-bit unless told otherwise, no cache and no
code shared with the package.  `forward(cfg, tensors, tokens)` returns the logits of every position (and, on request,
the residual stream after every layer); `tensors` maps the stored names to torch tensors, `cfg` is config.json as a dict.

Notation: W x for a stored matrix W [out, in]; t, j positions of one sequence counted from 0; h the input of a sublayer.

    stream         x_t = E[token_t] + P_t,   P_t[2i] = sin(t 10000^(-2i/width)),  P_t[2i+1] = cos of the same angle
    layer          x <- x + mixer(rms(x) (1 + w1)) ;  x <- x + ff(rms(x) (1 + w2))        (a layer may use an earlier one's tensors)
    mamba2         [z | x | B | C | dt] = W_in h;  x, B, C through a causal convolution per channel and silu;
                   S_t = exp(-exp(A_log) d_t) S_(t-1) + d_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,   d_t = softplus(dt_t + bias);
                   y silu(z), normed in equal parts, times a weight, W_o
    attention      two maps of causal windowed softmax attention per head over the same values, a1 - lambda a2,
                   divided by its root mean square over the head's values, times 1 - diff, W_o
    feed-forward   `top` of `experts` units down(relu(up h)^2), weighed by the softmax over the chosen logits, and a unit
                   for every token, weighed by the sigmoid of one number
    head           cap tanh(scale W rms(x) (1 + w) / cap)
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x, w, eps, dt):
    return rms(x, eps) * (1.0 + w.to(dt))


def silu(x):
    return x * torch.sigmoid(x)


def positions(T, width, dt, first=0):
    """The position vectors of `T` positions from `first` on."""
    out = torch.zeros(T, width, dtype=dt)
    for t in range(T):
        for c in range(width):
            angle = (first + t) * 10000.0 ** (-2.0 * (c // 2) / width)
            out[t, c] = math.sin(angle) if c % 2 == 0 else math.cos(angle)
    return out


def convolve(u, taps, bias):
    """u [T, C], taps [C, L] (the last column is the current token's): silu of the causal convolution with zeros before
    the start."""
    T, L = u.shape[0], taps.shape[1]
    out = bias.expand(T, -1).clone()
    for t in range(T):
        for j in range(L):
            if t - (L - 1) + j >= 0:
                out[t] += taps[:, j] * u[t - (L - 1) + j]
    return silu(out)


def state_space(x, B, C, d, a_log, skip):
    """x [T, H, V], B and C [T, G, N], d [T, H] (positive step sizes): y [T, H, V]."""
    T, H, V = x.shape
    G, N = B.shape[1:]
    y = torch.zeros_like(x)
    for h in range(H):
        g = h // (H // G)
        S = torch.zeros(N, V, dtype=x.dtype)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[h]) * d[t, h]) * S + d[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + skip[h] * x[t, h]
    return y


def gated_norm(y, z, parts, weight, eps):
    """y silu(z), divided by its root mean square in each of `parts` equal parts, times the weight."""
    T, I = y.shape
    v = (y * silu(z)).reshape(T, parts, I // parts)
    return rms(v, eps).reshape(T, I) * weight


def mamba2(m, tensors, pre, h, eps, dt):
    T = h.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    I = H * V
    W = lambda n: tensors[pre + n].to(dt)
    y = h @ W("in").T
    z, xbc, raw = y[:, :I], y[:, I:2 * I + 2 * G * N], y[:, 2 * I + 2 * G * N:]
    u = convolve(xbc, W("conv"), W("conv.b"))
    d = torch.logaddexp(raw + W("dt_bias"), torch.zeros((), dtype=dt))
    o = state_space(u[:, :I].reshape(T, H, V), u[:, I:I + G * N].reshape(T, G, N), u[:, I + G * N:].reshape(T, G, N), d,
                    W("A_log"), W("D"))
    return gated_norm(o.reshape(T, I), z, m["norm_groups"], W("norm"), eps) @ W("o").T


def one_map(q, k, v, scale, size):
    """q [H, T, D], k [H, T, D], v [H, T, V] (keys and values already one per query head)."""
    T = q.shape[1]
    t, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    visible = (j <= t) & (t - j < size)
    s = (q @ k.transpose(1, 2) * scale).masked_fill(~visible, float("-inf"))
    return torch.softmax(s, dim=-1) @ v


def difference(a1, a2, lam, diff, eps):
    """The two maps' outputs combined per head: [..., V]."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def mixing(tensors, pre, diff, dt):
    W = lambda n: tensors[pre + n].to(dt)
    return torch.exp((W("lq1") * W("lk1")).sum()) - torch.exp((W("lq2") * W("lk2")).sum()) + diff


def attention(m, tensors, pre, h, eps, dt):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    W = lambda n: tensors[pre + n].to(dt)
    q = (h @ W("q").T).reshape(T, H, 2, D)
    k = (h @ W("k").T).reshape(T, G, 2, D)
    v = (h @ W("v").T).reshape(T, G, V).permute(1, 0, 2).repeat_interleave(H // G, dim=0)
    maps = []
    for i in range(2):
        ki = k[:, :, i].permute(1, 0, 2).repeat_interleave(H // G, dim=0)
        maps.append(one_map(q[:, :, i].permute(1, 0, 2), ki, v, m["scale"], m["mask"]["size"]))
    o = difference(maps[0], maps[1], mixing(tensors, pre, m["diff"], dt), m["diff"], eps)
    return o.permute(1, 0, 2).reshape(T, H * V) @ W("o").T


def unit(tensors, pre, h, dt):
    W = lambda n: tensors[pre + n].to(dt)
    return torch.relu(h @ W("up").T) ** 2 @ W("down").T


def feed_forward(mlp, tensors, pre, h, dt, margins_out=None):
    """`margins_out`: a list that receives per token how far the last chosen logit lies above the first one left out (where
    that is tiny, a lower precision may choose otherwise)."""
    W = lambda n: tensors[pre + n].to(dt)
    E, top = mlp["router"]["experts"], mlp["router"]["top"]
    z = h @ W("router").T + W("router.b")
    if margins_out is not None and top < E:
        ranked = z.sort(dim=-1, descending=True).values
        margins_out.append(ranked[:, top - 1] - ranked[:, top])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = sorted(range(E), key=lambda e: (-float(z[t, e]), e))[:top]
        w = torch.softmax(z[t, chosen], dim=0)
        for i, e in enumerate(chosen):
            out[t] += w[i] * unit(tensors, f"{pre}e{e}.", h[t:t + 1], dt)[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ W("shared.sg").T) * unit(tensors, pre + "shared.", h, dt)
    return out


def head(x, tensors, scale, cap, dt):
    z = x @ tensors["head"].to(dt).T * scale
    return cap * torch.tanh(z / cap)


def forward(cfg, tensors, tokens, dt=torch.float64, layers_out=None, margins_out=None):
    eps = cfg["norm"]["eps"]
    x = tensors["embed"].to(dt)[torch.tensor(tokens, dtype=torch.long)] + positions(len(tokens), cfg["width"], dt)
    for i, layer in enumerate(cfg["layers"]):
        pre, m = f"l{layer.get('weights_of', i)}.", layer["mixer"]
        mixer = {"mamba2": mamba2, "attention": attention}[layer["type"]]
        x = x + mixer(m, tensors, pre + "mix.", norm(x, tensors[pre + "norm1"], eps, dt), eps, dt)
        if layer["mlp"] is not None:
            x = x + feed_forward(layer["mlp"], tensors, pre + "mlp.", norm(x, tensors[pre + "norm2"], eps, dt), dt, margins_out)
        if layers_out is not None:
            layers_out.append(x.clone())
    return head(norm(x, tensors["final.norm"], eps, dt), tensors, cfg["logit_scale"], cfg["logit_softcap"], dt)
