"""Small Soluzen configurations and random weights for the tests.  Weights are bf16 numbers, so that both dtypes of the
model and the fp64 restatement work on the same ones."""
import numpy as np
import torch


def attention(heads=3, dim=24, rot_dim=8, vdim=40, q_rank=20, kv_rank=36, window=7, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
            "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim},
            "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}


def mamba(heads=6, vdim=20, state=12, groups=3, conv=3, norm_groups=2):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def layer(mixer, ff=None):
    return {"type": "latent_attention" if "kv_rank" in mixer else "mamba2", "mixer": mixer,
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width, vocab, side, loop=None, eps=1e-5):
    c = {"architecture": "Soluzen", "layers": layers, "norm": {"eps": eps}, "token_side": {"dim": side}, "vocab": vocab, "width": width}
    if loop is not None:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


CASES = {
    # nothing a multiple of 8, a loop from the first layer on, a feed-forward behind a recurrence and none behind attention
    "odd": config([layer(mamba(), 52), layer(attention()), layer(mamba(heads=5, vdim=19, state=9, groups=1, conv=4, norm_groups=5)),
                   layer(attention(heads=2, dim=10, rot_dim=6, vdim=11, q_rank=13, kv_rank=17, window=19, base=500.0), 31)],
                  width=74, vocab=101, side=12, loop=(0, 3, 3)),
    # the sizes that the tensor-core kernels take, two kinds of attention
    "even": config([layer(attention(heads=2, dim=128, rot_dim=64, vdim=128, q_rank=96, kv_rank=256, window=70), 192),
                    layer(mamba(heads=4, vdim=32, state=64, groups=2, conv=4, norm_groups=4)),
                    layer(mamba(heads=3, vdim=80, state=128, groups=1, conv=2, norm_groups=1), 64),
                    layer(attention(heads=5, dim=40, rot_dim=16, vdim=72, q_rank=64, kv_rank=104, window=33), 136)],
                   width=128, vocab=264, side=16, loop=(1, 3, 2)),
    # no loop, a window of one, one tap, a group per head
    "plain": config([layer(attention(window=1), 40), layer(mamba(heads=4, vdim=8, state=8, groups=4, conv=1, norm_groups=4))],
                    width=48, vocab=64, side=8),
    # a loop that ends with the last layer, many passes
    "tail": config([layer(mamba(heads=2, vdim=16, state=16, groups=2, conv=5, norm_groups=1)), layer(attention(window=12), 24)],
                   width=40, vocab=50, side=4, loop=(1, 2, 4), eps=1e-3),
}


def shapes(cfg):
    w, n = cfg["width"], len(cfg["layers"])
    dim = cfg["token_side"]["dim"]
    s = {"embed": (cfg["vocab"], w), "side.embed": (cfg["vocab"], n * dim), "final.norm": (w,), "final.norm.b": (w,), "head": (cfg["vocab"], w)}
    if "loop" in cfg:
        s["loop.in"], s["loop.step"] = (w, 2 * w), (cfg["loop"]["times"], w)
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        s[p + "norm1"], s[p + "norm1.b"] = (w,), (w,)
        if lay["mlp"] is not None:
            ff = lay["mlp"]["ff"]
            s.update({p + "norm2": (w,), p + "norm2.b": (w,), p + "mlp.gate": (ff, w), p + "mlp.up": (ff, w), p + "mlp.down": (w, ff)})
        s.update({p + "side.gate": (dim, w), p + "side.proj": (w, dim), p + "side.norm": (w,)})
        p += "mix."
        if lay["type"] == "latent_attention":
            H, d, r, v, qr, kr = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            s.update({p + "dq": (qr, w), p + "dq.norm": (qr,), p + "uq": (H * (d + r), qr), p + "dkv": (kr + r, w), p + "dkv.norm": (kr,),
                      p + "uk": (H * d, kr), p + "uv": (H * v, kr), p + "o": (w, H * v)})
        else:
            H, v, N, G = (m[k] for k in ("heads", "vdim", "state", "groups"))
            C = H * v + 2 * G * N
            s.update({p + "in": (H * v + C + H, w), p + "conv": (C, m["conv"]), p + "conv.b": (C,), p + "dt_bias": (H,), p + "A_log": (H,),
                      p + "D": (H,), p + "norm": (H * v,), p + "o": (w, H * v)})
    return s


def weights(cfg, seed=0, peak=2.5):
    """name -> CPU bf16 tensor.  `peak` scales the query expansions: sharp attention, so that a single wrong key shows."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        x = rng.standard_normal(shape)
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith("side.norm"):
            x = 0.3 + 0.1 * x                      # what is added is normalised: a full-size one would drown the rest
        elif name.endswith("norm") or leaf in ("norm1", "norm2"):
            x = 1.0 + 0.3 * x
        elif leaf == "b":
            x = 0.2 * x
        elif leaf == "A_log":
            x = -1.5 + 1.5 * x                     # fast and slow heads
        elif leaf == "dt_bias":
            x = -1.5 + x
        elif leaf == "D":
            x = 1.0 + 0.3 * x
        elif leaf == "conv":
            x = x * 0.7
        elif leaf == "uq":
            x = peak * x / np.sqrt(shape[1])
        elif name == "loop.in":                    # mostly keeps the stream, mixes some of the embedding in
            x = 0.3 * x / np.sqrt(shape[1]) + np.eye(*shape)
        elif leaf in ("embed", "step"):
            x = x * (1.0 if leaf == "embed" else 0.3)
        else:
            x = x / np.sqrt(shape[-1])
        out[name] = torch.from_numpy(x.astype(np.float32)).to(torch.bfloat16)
    return out


def as_f64(w):
    return {k: v.double().numpy() for k, v in w.items()}


def row_errors(got, want):
    """Root mean square of the difference of each row, mean taken off, over that of `want`."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    s = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((s * s).mean())


def error(got, want):
    """The largest of them."""
    return float(row_errors(got, want).max())
