"""Plain numpy restatement of the Duponex decoder (fp64 unless a caller passes fp32 arrays): one function per mechanism,
whole sequences, no cache, no blocking.  The GPU tests compare the product path with it; it shares no code with the
package.

`weights` is a dict name -> array, `config` the parsed config.json.  A token sequence is always one 1-D array.
"""
from __future__ import annotations

import numpy as np


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def enter_streams(x, n):
    """(T, width) -> n equal copies, (n, T, width)."""
    return np.stack([x] * n)


def read_streams(streams, w_in):
    """What a sublayer reads: the weighted sum of the streams."""
    return np.einsum("s,stw->tw", w_in, streams)


def write_streams(streams, mix, w_out, y):
    """New stream t = sum over s of mix[s, t] (from s, to t) times old stream s, plus w_out[t] y."""
    return np.einsum("st,snw->tnw", mix, streams) + w_out[:, None, None] * y


def chunk_visible(T, size):
    """(T, T) bool: row i sees column j if j <= i and both lie in the same chunk of `size` positions."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def chunked_attention(q, k, v, scale, size):
    """q (T, H, E), k (T, G, E), v (T, G, V): query head h reads key / value head h // (H / G)."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    visible = chunk_visible(T, size)
    out = np.empty((T, H, v.shape[2]), dtype=np.result_type(q, v))
    for h in range(H):
        s = np.where(visible, (q[:, h] @ k[:, h // group].T) * scale, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h // group]
    return out


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, w, m, eps, v_first):
    """h (T, width); w(name) gives this mixer's tensors; m its sizes.  `v_first`: the values of the first layer that mixes,
    None in that layer itself.  Returns (output, values before mixing)."""
    T = h.shape[0]
    H, G, E, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w("q").T + w("q.b")).reshape(T, H, E), eps)
    k = unit_rms((h @ w("k").T + w("k.b")).reshape(T, G, E), eps)
    own = (h @ w("v").T + w("v.b")).reshape(T, G, V)
    v = own if not m["v_mix"] or v_first is None else mix_values(own, v_first, w("vmix"))
    o = chunked_attention(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, H * V)
    return (o * sigmoid(h @ w("g").T)) @ w("o").T + w("o.b"), own


def squared_relu_mlp(h, up, down):
    return squared_relu(h @ up.T) @ down.T


def forward(config, weights, tokens, layers_out=None):
    """tokens (T,) -> logits (T, vocab); `layers_out` (a list) receives the sum of the streams after every layer."""
    W = weights
    eps, mult = config["norm"]["eps"], config["residual_mult"]
    streams = enter_streams(W["embed"][np.asarray(tokens)] * config["embedding"]["scale"], config["streams"])
    v_first = None

    def sublayer(streams, p, q, f):
        u = read_streams(streams, W[f"{p}hc{q}.in"])
        y = f(rms_norm(u, W[f"{p}norm{q}"], eps)) * W[f"{p}ls{q}"]
        return write_streams(streams, W[f"{p}hc{q}.mix"], mult * W[f"{p}hc{q}.out"], y)

    for i, lay in enumerate(config["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        own = [None]

        def mixer(h):
            y, own[0] = attention(h, lambda s: W[p + "mix." + s], m, eps, v_first)
            return y
        streams = sublayer(streams, p, 1, mixer)
        if m["v_mix"] and v_first is None:
            v_first = own[0]
        if lay["mlp"] is not None:
            streams = sublayer(streams, p, 2, lambda h: squared_relu_mlp(h, W[p + "mlp.up"], W[p + "mlp.down"]))
        if layers_out is not None:
            layers_out.append(streams.sum(axis=0))
    return rms_norm(streams.sum(axis=0), W["final.norm"], eps) @ W["head"].T
