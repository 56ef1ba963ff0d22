"""Small Duponex configurations and random weights for the tests.  Weights are bf16 numbers, so that both dtypes of the model
and the fp64 restatement work on the same ones."""
import numpy as np
import torch

from soluzen_cases import as_f64, error, row_errors  # noqa: F401  (the error measures are the same)


def attention(heads=6, kv_heads=2, dim=10, vdim=11, chunk=7, v_mix=True, peak=3.0, scale=None):
    """`peak`: how sharp the attention is.  Queries and keys have unit RMS, so a score q.k has a spread of sqrt(dim)."""
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "v_mix": v_mix,
            "scale": peak * dim ** -0.5 if scale is None else scale}


def layer(mixer, ff=None):
    return {"type": "attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width, vocab, streams, mult=0.7, embed=0.5, eps=1e-5):
    return {"architecture": "Duponex", "embedding": {"scale": embed}, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult,
            "streams": streams, "vocab": vocab, "width": width}


CASES = {
    # nothing a multiple of 8, a layer that mixes no values between two that do, layers without a feed-forward
    "odd": config([layer(attention(), 52), layer(attention(heads=3, kv_heads=3, dim=5, vdim=9, chunk=19, v_mix=False)),
                   layer(attention(heads=2, dim=13, chunk=16), 31), layer(attention(heads=4, chunk=5))],
                  width=74, vocab=101, streams=3, mult=0.55, embed=1.7),
    # sizes of the tensor-core kernels; more than 16 query heads to a key head in one layer
    "even": config([layer(attention(heads=8, dim=64, vdim=128, chunk=70), 192),
                    layer(attention(heads=20, kv_heads=1, dim=32, vdim=40, chunk=33, v_mix=False), 136),
                    layer(attention(heads=2, dim=128, vdim=128, chunk=96))], width=128, vocab=264, streams=2),
    # one stream, chunks of one, a key head per query head, every constant 1
    "plain": config([layer(attention(heads=2, kv_heads=2, dim=16, vdim=8, chunk=1, v_mix=False, scale=1.0), 40),
                     layer(attention(heads=2, kv_heads=2, dim=16, vdim=8, chunk=1, v_mix=False, scale=1.0))],
                    width=48, vocab=64, streams=1, mult=1.0, embed=1.0),
    # the first layer that mixes values is not the first layer, wide heads, more streams than the register kernels take,
    # chunks longer than the sequences
    "wide": config([layer(attention(heads=2, kv_heads=1, dim=24, vdim=16, chunk=64, v_mix=False), 64),
                    layer(attention(heads=3, kv_heads=1, dim=200, vdim=136, chunk=500), 24),
                    layer(attention(heads=5, kv_heads=1, dim=72, vdim=136, chunk=40))], width=96, vocab=50, streams=5, eps=1e-3),
}


def shapes(cfg):
    w, n = cfg["width"], cfg["streams"]
    s = {"embed": (cfg["vocab"], w), "final.norm": (w,), "head": (cfg["vocab"], w)}
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        H, G, E, V = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
        for q in ("1", "2") if lay["mlp"] is not None else ("1",):
            s.update({p + "norm" + q: (w,), p + "ls" + q: (w,), f"{p}hc{q}.in": (n,), f"{p}hc{q}.out": (n,), f"{p}hc{q}.mix": (n, n)})
        s.update({p + "mix.q": (H * E, w), p + "mix.q.b": (H * E,), p + "mix.k": (G * E, w), p + "mix.k.b": (G * E,),
                  p + "mix.v": (G * V, w), p + "mix.v.b": (G * V,), p + "mix.g": (H * V, w), p + "mix.o": (w, H * V), p + "mix.o.b": (w,)})
        if m["v_mix"]:
            s[p + "mix.vmix"] = ()
        if lay["mlp"] is not None:
            s.update({p + "mlp.up": (lay["mlp"]["ff"], w), p + "mlp.down": (w, lay["mlp"]["ff"])})
    return s


def weights(cfg, seed=0):
    """name -> CPU bf16 tensor"""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        x = rng.standard_normal(shape)
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2", "ls1", "ls2"):
            x = 1.0 + 0.3 * x
        elif leaf == "b":
            x = 0.3 * x
        elif leaf == "vmix":
            x = rng.uniform(0.25, 0.75, shape)
        elif leaf == "in":
            x = rng.uniform(0.2, 1.0, shape)
        elif leaf == "out":
            x = 1.0 + 0.3 * x
        elif leaf == "mix" and len(shape) == 2:
            x = 0.9 * np.eye(shape[0]) + 0.15 * x
        elif leaf == "g":
            x = 2.0 * x / np.sqrt(shape[-1])
        elif leaf != "embed":
            x = x / np.sqrt(shape[-1])
        out[name] = torch.from_numpy(np.asarray(x, dtype=np.float32)).to(torch.bfloat16)
    return out
