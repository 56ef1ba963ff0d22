"""Plain numpy restatement of the Soluzen decoder (fp64 unless a caller passes fp32 arrays): one function per
mechanism, whole sequences, no cache, no blocking.  The GPU tests compare the product path with it; it shares no code
with the package.

`weights` is a dict name -> array, `config` the parsed config.json.  A token sequence is always one 1-D array.
"""
from __future__ import annotations

import math

import numpy as np


def layer_norm(x, w, b, eps):
    c = x - x.mean(axis=-1, keepdims=True)
    return c / np.sqrt((c * c).mean(axis=-1, keepdims=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def rotate_interleaved(x, positions, base):
    """x (T, ..., R): pair (2i, 2i+1) turned by positions * base**(-2i/R)."""
    R = x.shape[-1]
    f = float(base) ** (-np.arange(0, R, 2, dtype=np.float64) / R)
    a = np.asarray(positions, dtype=np.float64)[:, None] * f
    a = a.reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (R // 2,))
    u, v = x[..., 0::2], x[..., 1::2]
    out = np.empty_like(x)
    out[..., 0::2] = u * np.cos(a) - v * np.sin(a)
    out[..., 1::2] = v * np.cos(a) + u * np.sin(a)
    return out


def windowed_softmax_attention(q, k, v, scale, window):
    """q (T, H, E), k (T, H, E), v (T, H, V): position i sees the `window` positions that end at i."""
    T, H, _ = q.shape
    i = np.arange(T)[:, None]
    j = np.arange(T)[None, :]
    visible = (j <= i) & (i - j < window)
    out = np.empty((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = np.where(visible, (q[:, h] @ k[:, h].T) * scale, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h]
    return out


def latent_attention(h, w, m, eps):
    """h (T, width); w(name) gives this mixer's tensors; m its sizes."""
    T = h.shape[0]
    H, d, r, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    cq = rms_norm(h @ w("dq").T, w("dq.norm"), eps)
    q = (cq @ w("uq").T).reshape(T, H, d + r)
    ckv = h @ w("dkv").T
    c = rms_norm(ckv[:, :kr], w("dkv.norm"), eps)
    base = m["rot"]["base"]
    k_rot = rotate_interleaved(ckv[:, kr:], pos, base)
    q = np.concatenate([q[:, :, :d], rotate_interleaved(q[:, :, d:], pos, base)], axis=2)
    k = np.concatenate([(c @ w("uk").T).reshape(T, H, d), np.repeat(k_rot[:, None], H, axis=1)], axis=2)
    v = (c @ w("uv").T).reshape(T, H, dv)
    o = windowed_softmax_attention(q, k, v, m["scale"], m["mask"]["size"])
    return o.reshape(T, H * dv) @ w("o").T


def causal_conv(x, taps, bias):
    """x (T, C), taps (C, K): the last column multiplies the current token; zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = np.tile(bias, (T, 1)).astype(x.dtype)
    for k in range(K):
        back = K - 1 - k
        y[back:] += x[:T - back if back else T] * taps[:, k] if back < T else 0.0
    return y


def selective_scan(x, B, C, dt, A, D):
    """x (T, H, P), B and C (T, G, N), dt (T, H), A and D (H): the linear recurrence, token by token."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, P), dtype=x.dtype)
    group = np.arange(H) // (H // G)
    y = np.empty_like(x)
    for t in range(T):
        b, c = B[t][group], C[t][group]
        S = np.exp(A * dt[t])[:, None, None] * S + dt[t][:, None, None] * b[:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnp,hn->hp", S, c) + D[:, None] * x[t]
    return y


def gated_group_norm(y, z, w, groups, eps):
    T, n = y.shape
    g = (y * silu(z)).reshape(T, groups, n // groups)
    g = g / np.sqrt((g * g).mean(axis=2, keepdims=True) + eps)
    return g.reshape(T, n) * w


def mamba2(h, w, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    zxbcdt = h @ w("in").T
    z = zxbcdt[:, :inner]
    xbc = silu(causal_conv(zxbcdt[:, inner:2 * inner + 2 * G * N], w("conv"), w("conv.b")))
    dt = softplus(zxbcdt[:, 2 * inner + 2 * G * N:] + w("dt_bias"))
    y = selective_scan(xbc[:, :inner].reshape(T, H, P), xbc[:, inner:inner + G * N].reshape(T, G, N),
                       xbc[:, inner + G * N:].reshape(T, G, N), dt, -np.exp(w("A_log")), w("D"))
    return gated_group_norm(y.reshape(T, inner), z, w("norm"), m["norm_groups"], eps) @ w("o").T


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2}


def gated_mlp(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def token_side(x, e, gate, proj, norm, eps):
    y = (gelu_tanh(x @ gate.T) * e) @ proj.T
    return rms_norm(y, norm, eps)


def schedule(config):
    """The layer runs in order: (layer, pass of the loop that starts here or None)."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(config, weights, tokens, layers_out=None):
    """tokens (T,) -> logits (T, vocab); `layers_out` (a list) receives the residual stream after every layer run."""
    W = weights
    tokens = np.asarray(tokens)
    eps = config["norm"]["eps"]
    x = x0 = W["embed"][tokens]
    side = W["side.embed"][tokens]
    dim = config["token_side"]["dim"]

    def norm(name, v):
        return layer_norm(v, W[name], W[name + ".b"], eps)

    for i, start_of_pass in schedule(config):
        if start_of_pass is not None:
            x = np.concatenate([x, x0], axis=1) @ W["loop.in"].T + W["loop.step"][start_of_pass]
        lay, p = config["layers"][i], f"l{i}."
        x = x + MIXERS[lay["type"]](norm(p + "norm1", x), lambda s: W[p + "mix." + s], lay["mixer"], eps)
        if lay["mlp"] is not None:
            x = x + gated_mlp(norm(p + "norm2", x), W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"])
        x = x + token_side(x, side[:, i * dim:(i + 1) * dim], W[p + "side.gate"], W[p + "side.proj"], W[p + "side.norm"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return norm("final.norm", x) @ W["head"].T
