"""Plain statement of the Tibalorn decoder for the tests: one function per mechanism, one sequence at a time, written with
torch in one precision (float64 unless a caller asks for less), with loops over tokens where the definition is a recurrence.
Slow on purpose and independent of the package: it imports nothing from ``sneppx_alg_b200``.

Shapes: activations [T, channels], heads split as [T, heads, size]. Weights are the checkpoint's tensors by name."""
from __future__ import annotations

import math

import torch


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def squared_relu(x):
    return torch.clamp(x, min=0) ** 2


def softcap(x, cap):
    return cap * torch.tanh(x / cap)


def layer_norm(x, w, b, eps):
    m = x.mean(-1, keepdim=True)
    var = ((x - m) ** 2).mean(-1, keepdim=True)
    return (x - m) / torch.sqrt(var + eps) * w + b


def group_rms(y, groups, eps, w):
    """RMS norm of ``groups`` equal parts of every row, each by its own mean square."""
    T, n = y.shape
    p = y.view(T, groups, n // groups)
    return (p / torch.sqrt((p * p).mean(-1, keepdim=True) + eps)).reshape(T, n) * w


def short_conv(u, w, b):
    """y_t = b + sum_j w[:, j] u_{t - taps + 1 + j}; the last column meets the current token."""
    T, taps = u.shape[0], w.shape[1]
    y = b[None].repeat(T, 1)
    for j in range(taps):
        back = taps - 1 - j
        y[back:] += w[:, j] * u[:T - back] if back < T else 0
    return y


# ------------------------------------------------------------------------------------------------ rotation
def rotary_frequencies(dims, base, scaling=None):
    """Frequency of every pair and the factor on cos and sin; ``scaling`` stretches the slow pairs (YaRN)."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1


def rotate_half(x, freqs, mul=1.0, sign=1, start=0):
    """Pairs (i, i + n) of the first 2 n entries of every head turn by sign * position * freqs[i]; x [T, heads, size]."""
    n = len(freqs)
    if n == 0:
        return x.clone()
    pos = torch.arange(start, start + x.shape[0], dtype=torch.float64)
    a = sign * pos[:, None] * torch.tensor(freqs, dtype=torch.float64)
    c, s = (torch.cos(a) * mul).to(x.dtype)[:, None], (torch.sin(a) * mul).to(x.dtype)[:, None]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


# ------------------------------------------------------------------------------------------------ attention
def token_visible(i, j, size):
    return 0 <= i - j < size


def block_visible(i, b, pool, size):
    return (b + 1) * pool - 1 <= i - size


def pooled_window_attention(q, k, v, scale, temp, sink, size, pool, at=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]: the last ``size`` tokens one by one, earlier ones as means of
    whole blocks of ``pool`` tokens, one softmax with exp(sink[h]) added to its denominator. ``at``: only these positions (the others stay
    zero)."""
    T, H, _ = q.shape
    G, NB = k.shape[1], T // pool
    kb = k[:NB * pool].view(NB, pool, *k.shape[1:]).mean(1)
    vb = v[:NB * pool].view(NB, pool, *v.shape[1:]).mean(1)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in (range(T) if at is None else at):
        js = [j for j in range(max(0, i - size + 1), i + 1) if token_visible(i, j, size)]
        bs = [b for b in range(NB) if block_visible(i, b, pool, size)]
        kk, vv = torch.cat([k[js], kb[bs]]), torch.cat([v[js], vb[bs]])
        for h in range(H):
            g = h // (H // G)
            s = (kk[:, g] @ q[i, h]) * scale * temp[h]
            m = torch.maximum(s.max(), sink[h])
            e = torch.exp(s - m)
            out[i, h] = (e[:, None] * vv[:, g]).sum(0) / (e.sum() + torch.exp(sink[h] - m))
    return out


# ------------------------------------------------------------------------------------------------ recurrence
def ssd(x, B, C, dt, A_log, D, S=None):
    """x [T, H, P], B, C [T, G, N], dt [T, H] -> y [T, H, P], S [H, N, P]: decay, write dt B x^T, read with C."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype) if S is None else S.clone()
    own = [h // (H // G) for h in range(H)]
    y = torch.zeros_like(x)
    for t in range(T):
        a = torch.exp(-torch.exp(A_log) * dt[t])
        S = a[:, None, None] * S + dt[t][:, None, None] * B[t, own][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t, own][:, :, None]).sum(1) + D[:, None] * x[t]
    return y, S


# ------------------------------------------------------------------------------------------------ mixers
def mamba2_mixer(h, W, p, c, eps):
    T, H, P, N, G = h.shape[0], c["heads"], c["vdim"], c["state"], c["groups"]
    inner = H * P
    u = h @ W[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner: 2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = xbc[:, :inner].view(T, H, P), xbc[:, inner: inner + G * N].view(T, G, N), xbc[:, inner + G * N:].view(T, G, N)
    y, _ = ssd(x, B, C, softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"])
    return group_rms(y.reshape(T, inner) * silu(z), c["norm_groups"], eps, W[p + "norm"]) @ W[p + "o"].T


def attention_mixer(h, W, p, c, eps):
    T, H, G, d, dv, rot = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["rot"]
    q, k, v = (h @ W[p + n].T + W[p + n + ".b"] for n in "qkv")
    freqs, mul = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    q, k = rotate_half(q.view(T, H, d), freqs, mul), rotate_half(k.view(T, G, d), freqs, mul)
    vfreqs, _ = rotary_frequencies(dv, rot["base"])
    v = rotate_half(v.view(T, G, dv), vfreqs)
    o = pooled_window_attention(q, k, v, c["scale"], W[p + "temp"], W[p + "sink"], c["mask"]["size"], c["mask"]["pool"])
    o = rotate_half(o, vfreqs, sign=-1).reshape(T, H * dv)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


MIXERS = {"mamba2": mamba2_mixer, "attention": attention_mixer}


def forward(cfg, W, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence. ``layers_out``: list that receives the residual stream after each layer."""
    W = {k: t.to(dtype) for k, t in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[spec["type"]](layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps), W, p + "mix.", spec["mixer"], eps)
        if spec["mlp"] is not None:
            a = layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps) @ W[p + "mlp.up"].T
            x = x + squared_relu(a) @ W[p + "mlp.down"].T
        if layers_out is not None:
            layers_out.append(x.clone())
    return softcap(layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["embed"].T, cfg["logit_softcap"])
