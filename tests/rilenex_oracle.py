"""Plain statement of the Rilenex decoder for the tests: one function per mechanism, one sequence at a time, written
with torch in one precision (float64 unless a caller asks for less) and loops over tokens where the definition is a
recurrence. Slow on purpose and independent of the package: it imports nothing from ``sneppx_alg_b200``.

Shapes: activations [T, channels], heads split as [T, heads, size]. Weights are the checkpoint's tensors by name."""
from __future__ import annotations

import torch


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def xielu(z, p, q):
    """Piecewise activation: quadratic growth above zero, bounded exponential below, slope 1/2 at zero."""
    pos = softplus(p) * z * z + 0.5 * z
    zn = torch.clamp(z, max=0)
    neg = (0.5 + softplus(q)) * (torch.exp(zn) - 1 - zn) + 0.5 * z
    return torch.where(z > 0, pos, neg)


def short_conv(u, w):
    """y_t = sum_j w[:, j] u_{t - taps + 1 + j}; the last column meets the current token."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def rotate(x, dims, base, start=0):
    """Interleaved rotation of the first ``dims`` entries of every head; x [T, heads, size], positions from start."""
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = torch.tensor(float(start + t), dtype=torch.float64) * float(base) ** (-2.0 * i / dims)
            c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            out[t, :, 2 * i] = u * c - v * s
            out[t, :, 2 * i + 1] = v * c + u * s
    return out


def chunk_visible(i, j, size):
    return j <= i and i // size == j // size


def talking_attention(q, k, v, scale, talk, size):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]: raw scores, mixed over heads, softmax in the chunk."""
    T, H, _ = q.shape
    G = k.shape[1]
    kv = [h // (H // G) for h in range(H)]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        js = [j for j in range(T) if chunk_visible(i, j, size)]
        raw = torch.stack([k[js][:, kv[h]] @ q[i, h]
                           for h in range(H)]) * scale
        p = torch.softmax(talk @ raw, dim=-1)
        for h in range(H):
            out[i, h] = p[h] @ v[js][:, kv[h]]
    return out


def delta_rule(q, k, v, beta, g, S=None):
    """q, k [T, H, d], v [T, H, dv], beta [T, H], g [T, H, d] -> o [T, H, dv], S [H, d, dv]. Decay, error-correcting
    write, then read."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    o = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        for h in range(H):
            M = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - M.T @ k[t, h])
            S[h] = M + torch.outer(k[t, h], u)
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def gated_write(q, f, v, S=None):
    """q, f [T, H, d], v [T, H, dv]: S <- f S + (1 - f) v^T, o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    o = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        for h in range(H):
            S[h] = f[t, h][:, None] * S[h] + torch.outer(1 - f[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


# ------------------------------------------------------------------------------------------------ mixers
def hgrn2_mixer(h, W, p, c, eps):
    T, H, d, dv = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = silu(h @ W[p + "q"].T).view(T, H, d)
    v = (h @ W[p + "v"].T).view(T, H, dv)
    low = W[p + "lower"]
    f = (low + (1 - low) * sigmoid(h @ W[p + "f"].T + W[p + "f.b"])).view(T, H, d)
    o, _ = gated_write(q, f, v)
    return rms(o, eps, W[p + "norm"]).reshape(T, H * dv) @ W[p + "o"].T


def attention_mixer(h, W, p, c, eps):
    T, H, G, d, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (short_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q = rms(q.view(T, H, d), eps, W[p + "q.norm"])
    k = rms(k.view(T, G, d), eps, W[p + "k.norm"])
    rot = c["rot"]
    q, k = rotate(q, rot["dims"], rot["base"]), rotate(k, rot["dims"], rot["base"])
    o = talking_attention(q, k, v.view(T, G, dv), c["scale"], W[p + "talk"], c["mask"]["size"])
    o = o * sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ W[p + "o"].T


def delta_mixer(h, W, p, c, eps):
    T, H, G, d, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(short_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in "qkv")
    own = [i // (H // G) for i in range(H)]
    q = (unit(q.view(T, G, d)) * d ** -0.5)[:, own]
    k = unit(k.view(T, G, d))[:, own]
    beta = sigmoid(h @ W[p + "b"].T)
    raw = ((h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]).view(T, H, d)
    g = torch.exp(-torch.exp(W[p + "A_log"])[None, :, None] * softplus(raw))
    o, _ = delta_rule(q, k, v.view(T, H, dv), beta, g)
    gate = sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T)
    return (rms(o, eps, W[p + "norm"]).reshape(T, H * dv) * gate) @ W[p + "o"].T


def parallel_mixer(h, W, p, c, eps):
    return (c["left_scale"] * attention_mixer(h, W, p + "left.", c["left"], eps)
            + c["right_scale"] * delta_mixer(h, W, p + "right.", c["right"], eps))


MIXERS = {"hgrn2": hgrn2_mixer, "parallel": parallel_mixer}


def forward(cfg, W, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence. ``layers_out``: list that receives the residual stream after each layer."""
    W = {k: t.to(dtype) for k, t in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)]
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[spec["type"]](rms(x, eps, W[p + "norm1"]), W, p + "mix.", spec["mixer"], eps)
        if spec["mlp"] is not None:
            a = rms(x, eps, W[p + "norm2"]) @ W[p + "mlp.up"].T
            pq = W[p + "mlp.act"]
            x = x + xielu(a, pq[0], pq[1]) @ W[p + "mlp.down"].T
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, eps, W["final.norm"]) @ W["head"].T
