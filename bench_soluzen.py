"""Throughput of the Soluzen design at sizes that resemble a real model's layers, beside the LLaMA family at equal width:
`python bench.py --soluzen`.

Whole models (prompt pass, decode steps replayed from a CUDA graph) and every kernel of the design by itself, each against
its roofline.  A kernel is timed with CUDA events over a loop whose inputs together exceed the L2 (several sets of buffers
where one set would fit)."""
from __future__ import annotations

import torch

WIDTH, FF, VOCAB = 2048, 5632, 32000
ATTENTION = dict(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512, mask={"size": 1024},
                 rot={"base": 10000.0, "dims": 64}, scale=192 ** -0.5)
MAMBA = dict(heads=64, vdim=64, state=128, groups=1, conv=4, norm_groups=1)
SIDE = 256
L2_BYTES = 126e6


def config(window, n_blocks=2):
    """`n_blocks` x [attention + MLP, mamba2, mamba2, mamba2], a middle part run twice."""
    att = dict(ATTENTION, mask={"size": window})
    block = [{"type": "latent_attention", "mixer": att, "mlp": {"kind": "dense", "ff": FF}}] + \
            [{"type": "mamba2", "mixer": MAMBA, "mlp": None}] * 3
    n = 4 * n_blocks
    return {"architecture": "Soluzen", "layers": block * n_blocks, "loop": {"start": n // 2, "stop": n, "times": 2},
            "norm": {"eps": 1e-5}, "token_side": {"dim": SIDE}, "vocab": VOCAB, "width": WIDTH}


class RandomWeights:
    """A stand-in for a checkpoint: N(0, 0.02) of whatever shape is asked for, drawn on the GPU; norms are ones."""

    def __init__(self, seed=0):
        self.gen = torch.Generator(device="cuda").manual_seed(seed)

    def __call__(self, name, *shape):
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2"):
            return torch.ones(shape, device="cuda", dtype=torch.bfloat16)
        x = torch.randn(shape, generator=self.gen, device="cuda") * 0.02
        return (x - 2.0 if leaf == "dt_bias" else x).to(torch.bfloat16)

    def leftover(self):
        return []


def build(window, n_blocks=2):
    from baranet_bdml_b200 import _lib
    from baranet_bdml_b200.soluzen import SoluzenConfig, SoluzenModel
    _lib.load()
    return SoluzenModel(SoluzenConfig.from_dict(config(window, n_blocks)), RandomWeights())


def timed(fn, steps=20, warmup=3):
    for i in range(warmup):
        fn(i)
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for i in range(steps):
        fn(warmup + i)
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


def timed_graph(fn, steps=20, inner=8):
    """The same with `inner` launches per graph replay: for kernels shorter than their launch from Python."""
    for i in range(inner):
        fn(i)
    torch.cuda.synchronize()
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        fn(0)
    torch.cuda.current_stream().wait_stream(side)
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for i in range(inner):
            fn(i)
    return timed(lambda i: graph.replay(), steps) / inner


class Kernels:
    """Times single launches; entries are (ms, bound, achieved, fraction of the measured peak)."""

    def __init__(self, pk):
        self.pk, self.out = pk, {}

    def hbm(self, name, ms, nbytes):
        gbs = nbytes / ms * 1e-6
        self.out[name] = {"us": ms * 1e3, "bound": "HBM", "GB_per_s": gbs, "frac": gbs / self.pk["hbm"]}

    def tensor(self, name, ms, flops):
        tf = flops / ms * 1e-9
        self.out[name] = {"us": ms * 1e3, "bound": "tensor", "TFLOP_per_s": tf, "frac": tf / self.pk["tensor"]}


def prompt_kernels(pk, B=8, S=2048, window=1024):
    from baranet_bdml_b200 import _lib, ops
    from baranet_bdml_b200.soluzen import _mixer_config
    from baranet_bdml_b200.mixers import GatedMLP, LatentAttention, Mamba2Mixer, TokenSide
    lib, K, bf = _lib.load(), Kernels(pk), torch.bfloat16
    w = RandomWeights()
    get = lambda name, *shape: w(name, *shape)                                    # noqa: E731
    T = B * S
    st = lambda: torch.cuda.current_stream().cuda_stream                          # noqa: E731
    rnd = lambda *shape, dtype=bf: torch.randn(shape, device="cuda").to(dtype)    # noqa: E731
    at = LatentAttention(_mixer_config("latent_attention", dict(ATTENTION, mask={"size": window})), WIDTH, 1e-5, get, bf)
    mb = Mamba2Mixer(_mixer_config("mamba2", MAMBA), WIDTH, 1e-5, get, bf)
    c, m = at.cfg, mb.cfg
    seq, pos = torch.arange(B, dtype=torch.int32, device="cuda"), torch.zeros(B, dtype=torch.int32, device="cuda")
    h = rnd(T, WIDTH)

    def gemm(name, lin, x, **kw):
        K.tensor(name, timed(lambda i: lin(x, **kw)), 2.0 * T * lin.n * lin.k)
    gemm("product dq|dkv", at.down, h)
    gemm("product uq", at.uq, rnd(T, at.uq.k))
    gemm("product uk|uv", at.ukv, rnd(T, at.ukv.k))
    gemm("product o (attention)", at.o, rnd(T, at.o.k))
    gemm("product in (mamba2)", mb.proj_in, h)
    gemm("product o (mamba2)", mb.o, rnd(T, mb.o.k))
    mlp = GatedMLP(FF, WIDTH, "gelu_tanh", get, bf)
    K.tensor("gate/up with gelu", timed(lambda i: mlp.gate_up(h)), 2.0 * T * 2 * FF * WIDTH)
    gemm("product down", mlp.down, rnd(T, FF))
    side = TokenSide(SIDE, WIDTH, 1e-5, "gelu_tanh", get, bf)
    e = rnd(T, SIDE)
    # both products of the token input read and write more than they compute
    K.hbm("token gate with gelu * e", timed(lambda i: side.gate.act_mul(h, e, "gelu_tanh")), T * (WIDTH + 2 * SIDE) * 2 + SIDE * WIDTH * 2)
    K.hbm("token projection", timed(lambda i: side.proj(e)), T * (WIDTH + SIDE) * 2 + SIDE * WIDTH * 2)
    lin3 = ops.Linear(rnd(WIDTH, 3 * WIDTH), bf)
    gemm("pass input, fp32 result", lin3, rnd(T, 3 * WIDTH), f32_out=True)

    # attention
    proj = rnd(T, at.down.n)
    cq, lat, key = rnd(T, c.q_rank), rnd(T, at.kv_ld), rnd(T, at.rot_ld)
    cache = at.new_state(B)
    K.hbm("latent_prep", timed(lambda i: at._prep(proj, B, S, cache, seq, pos, lat, key, S, 0)),
          T * (2 * (c.q_rank + c.kv_rank + c.rot_dim)) * 2 + B * min(S, cache.ring_tokens) * (at.kv_ld + at.rot_ld) * 2)
    q, kv, out = rnd(T, at.uq.n), rnd(T, at.ukv.n), rnd(T, at.o.k)
    K.hbm("rope_heads", timed(lambda i: lib.bn_rope_heads(q.data_ptr(), q.stride(0), B, S, c.heads, c.dim, c.rot_dim, at.freq.data_ptr(),
                                                          pos.data_ptr(), 1, st())), 2 * T * c.heads * c.rot_dim * 2)
    seen = sum(min(i + 1, window) for i in range(S))

    def attn(i):
        _lib.check(lib.bn_attn_window(q.data_ptr(), q.stride(0), kv.data_ptr(), kv.data_ptr() + c.heads * c.dim * 2, kv.stride(0),
                                      key.data_ptr(), at.rot_ld, out.data_ptr(), out.stride(0), B, S, 0, S, c.heads, c.dim, c.rot_dim, c.vdim,
                                      window, float(c.scale), ops.status_word("cuda").data_ptr(), 1, st()))
    K.tensor(f"attn_portion_sm100, window {window}", timed(attn), 2.0 * B * c.heads * seen * (c.dim + c.rot_dim + c.vdim))

    # mamba2
    pin = rnd(T, mb.proj_in.n)
    rs = mb.new_state(B)
    xbc = rnd(T, ops.round8(m.channels))
    dt, a = torch.rand((T, m.heads), device="cuda") * 0.1, -torch.rand((T, m.heads), device="cuda") * 0.2
    y = rnd(T, m.inner)

    def conv(i):
        _lib.check(lib.bn_mamba2_conv(pin.data_ptr(), pin.stride(0), mb.conv.data_ptr(), mb.conv_bias.data_ptr(), mb.dt_bias.data_ptr(),
                                      mb.a_log.data_ptr(), rs.conv.data_ptr(), seq.data_ptr(), pos.data_ptr(), B, S, m.heads, m.vdim, m.groups,
                                      m.state, m.taps, xbc.data_ptr(), xbc.stride(0), dt.data_ptr(), a.data_ptr(), 1, st()))

    def scan(i):
        _lib.check(lib.bn_ssm_scan(xbc.data_ptr(), xbc.stride(0), dt.data_ptr(), a.data_ptr(), mb.d.data_ptr(), rs.state.data_ptr(), seq.data_ptr(),
                                   B, S, m.heads, m.vdim, m.groups, m.state, y.data_ptr(), y.stride(0), 1, st()))
    K.hbm("mamba2 conv + steps", timed(conv), T * (2 * m.channels * 2 + m.heads * (2 + 8)))
    ms = timed(scan)
    K.hbm("ssd_scan", ms, T * ((m.channels + m.inner) * 2 + m.heads * 8) + 2 * B * m.heads * m.vdim * m.state * 4)
    # products of a chunk of 64 tokens and a head: C B^T, M x, C S, w x B (the last three with two-part operands)
    K.out["ssd_scan"]["TFLOP_per_s"] = 2.0 * T * m.heads * (64 * m.state + 2 * 64 * m.vdim + 4 * m.state * m.vdim) / ms * 1e-9
    og = rnd(T, m.inner)
    K.hbm("gated_group_norm", timed(lambda i: lib.bn_gated_group_norm(y.data_ptr(), y.stride(0), 1, pin.data_ptr(), pin.stride(0), mb.norm.data_ptr(),
                                                                      og.data_ptr(), og.stride(0), T, m.inner, 1, 1e-5, 1, st())), 3 * T * m.inner * 2)

    # residual stream
    x = torch.randn((T, WIDTH), device="cuda")
    nw = ops.NormWeight(torch.ones(WIDTH), torch.zeros(WIDTH), 1e-5)
    cast = rnd(T, WIDTH)
    K.hbm("residual_norm: add, layer norm", timed(lambda i: ops.residual_norm(x, ops.Pending(h), bf, WIDTH, norm=nw)), T * WIDTH * (4 + 2 + 4 + 2))
    K.hbm("residual_norm: add normed, layer norm", timed(lambda i: ops.residual_norm(x, ops.Pending(h, side.norm), bf, WIDTH, norm=nw)),
          T * WIDTH * (4 + 2 + 4 + 2))
    K.hbm("residual_norm: add, rounded copy", timed(lambda i: ops.residual_norm(x, ops.Pending(h), bf, WIDTH, cast=cast)), T * WIDTH * (4 + 2 + 4 + 2))
    ids = torch.randint(0, VOCAB, (T,), device="cuda", dtype=torch.int32)
    table = rnd(VOCAB, WIDTH)
    K.hbm("embedding rows", timed(lambda i: ops.embedding_rows(table, ids, out_f32=x, out_bf16=cast)), T * WIDTH * 8)
    return K.out


def step_kernels(pk, B, window=4096):
    from baranet_bdml_b200 import _lib, ops
    from baranet_bdml_b200.soluzen import _mixer_config
    from baranet_bdml_b200.mixers import GatedMLP, LatentAttention, Mamba2Mixer, TokenSide
    lib, K, bf = _lib.load(), Kernels(pk), torch.bfloat16
    w = RandomWeights()
    get = lambda name, *shape: w(name, *shape)                                    # noqa: E731
    st = lambda: torch.cuda.current_stream().cuda_stream                          # noqa: E731
    rnd = lambda *shape, dtype=bf: torch.randn(shape, device="cuda").to(dtype)    # noqa: E731
    sets = 8
    acfg = _mixer_config("latent_attention", dict(ATTENTION, mask={"size": window}))
    ats = [LatentAttention(acfg, WIDTH, 1e-5, get, bf) for _ in range(sets)]
    mbs = [Mamba2Mixer(_mixer_config("mamba2", MAMBA), WIDTH, 1e-5, get, bf) for _ in range(sets)]
    at, mb = ats[0], mbs[0]
    c, m = at.cfg, mb.cfg
    seq = torch.arange(B, dtype=torch.int32, device="cuda")
    pos = torch.full((B,), 3 * window + 11, dtype=torch.int32, device="cuda")
    H, width = c.heads, at.kv_ld + at.rot_ld
    rings = [a.new_state(B) for a in ats]
    q_abs = rnd(B, H, width)
    splits = lib.bn_latent_decode_splits(B, H, c.kv_rank, c.rot_dim, window, 1)
    part, lse = torch.zeros((B, H, splits, at.kv_ld), device="cuda"), torch.zeros((B, H, splits), device="cuda")

    def attend(i):
        r = rings[i % sets]
        _lib.check(lib.bn_latent_decode(q_abs.data_ptr(), r.ring.data_ptr(), B, r.ring_tokens, seq.data_ptr(), pos.data_ptr(), part.data_ptr(),
                                        lse.data_ptr(), splits, B, H, c.kv_rank, c.rot_dim, window, float(c.scale), 1, st()))
    K.hbm(f"latent_decode, window {window}", timed_graph(attend), B * window * width * 2)
    K.out[f"latent_decode, window {window}"]["splits"] = splits
    q, out = rnd(B, at.uq.n), rnd(B, at.o.k)
    K.hbm("latent_absorb_q", timed_graph(lambda i: lib.bn_latent_absorb_q(q.data_ptr(), q.stride(0), ats[i % sets].uk.data_ptr(), at.freq.data_ptr(),
                                                                          pos.data_ptr(), q_abs.data_ptr(), B, H, c.dim, c.rot_dim, c.kv_rank, 1, st())),
          H * c.dim * at.kv_ld * 2 + B * H * (c.dim + c.rot_dim + width) * 2)
    K.hbm("latent_expand_out", timed_graph(lambda i: lib.bn_latent_expand_out(part.data_ptr(), lse.data_ptr(), splits, ats[i % sets].uv.data_ptr(),
                                                                              out.data_ptr(), out.stride(0), B, H, c.vdim, c.kv_rank, 1, st())),
          H * c.vdim * at.kv_ld * 2 + B * H * (splits * at.kv_ld * 4 + c.vdim * 2))
    proj = rnd(B, at.down.n)
    K.hbm("latent_prep", timed_graph(lambda i: ats[i % sets]._prep(proj, B, 1, rings[i % sets], seq, pos, None, None, 0, 0)),
          B * 2 * at.down.n * 2)
    states = [x.new_state(B) for x in mbs]
    pin, gated = rnd(B, mb.proj_in.n), torch.zeros((B, m.inner), device="cuda")

    def step(i):
        s, x = states[i % sets], mbs[i % sets]
        _lib.check(lib.bn_mamba2_step(pin.data_ptr(), pin.stride(0), x.conv.data_ptr(), x.conv_bias.data_ptr(), x.dt_bias.data_ptr(), x.a_log.data_ptr(),
                                      x.d.data_ptr(), s.conv.data_ptr(), s.state.data_ptr(), seq.data_ptr(), pos.data_ptr(), B, m.heads, m.vdim, m.groups,
                                      m.state, m.taps, gated.data_ptr(), 1, st()))
    K.hbm("mamba2_step", timed_graph(step), B * m.heads * m.vdim * m.state * 8 + B * (mb.proj_in.n * 2 + m.inner * 4 + m.channels * m.taps * 2))
    og = rnd(B, m.inner)
    K.hbm("gated_group_norm", timed_graph(lambda i: lib.bn_gated_group_norm(gated.data_ptr(), m.inner, 0, None, 0, mb.norm.data_ptr(), og.data_ptr(),
                                                                            og.stride(0), B, m.inner, 1, 1e-5, 1, st())), B * m.inner * 6)
    mlps = [GatedMLP(FF, WIDTH, "gelu_tanh", get, bf) for _ in range(sets)]
    sides = [TokenSide(SIDE, WIDTH, 1e-5, "gelu_tanh", get, bf) for _ in range(sets)]
    h, e = rnd(B, WIDTH), rnd(B, SIDE)

    def weight_stream(name, fn, lin, extra=1):
        K.hbm(name, timed_graph(fn), extra * lin.n * lin.k * 2 + B * (lin.n + lin.k) * 2)
    weight_stream("product dq|dkv", lambda i: ats[i % sets].down(h), at.down)
    cq = rnd(B, at.uq.k)
    weight_stream("product uq", lambda i: ats[i % sets].uq(cq), at.uq)
    weight_stream("product o (attention)", lambda i: ats[i % sets].o(out), at.o)
    weight_stream("product in (mamba2)", lambda i: mbs[i % sets].proj_in(h), mb.proj_in)
    weight_stream("product o (mamba2)", lambda i: mbs[i % sets].o(og), mb.o)
    weight_stream("gate/up with gelu", lambda i: mlps[i % sets].gate_up(h), mlps[0].gate_up.gate, 2)
    hf = rnd(B, FF)
    weight_stream("product down", lambda i: mlps[i % sets].down(hf), mlps[0].down)
    weight_stream("token gate with gelu * e", lambda i: sides[i % sets].gate.act_mul(h, e, "gelu_tanh"), sides[0].gate)
    weight_stream("token projection", lambda i: sides[i % sets].proj(e), sides[0].proj)
    x = torch.randn((B, WIDTH), device="cuda")
    nw = ops.NormWeight(torch.ones(WIDTH), torch.zeros(WIDTH), 1e-5)
    K.hbm("residual_norm: add, layer norm", timed_graph(lambda i: ops.residual_norm(x, ops.Pending(h), bf, WIDTH, norm=nw)), B * WIDTH * 12)
    return K.out


def llama_step_kernels(pk, B):
    """The LLaMA family's kernels for the same step, timed the same way: what a short launch can reach."""
    from baranet_bdml_b200 import layers as L, ops
    K, bf = Kernels(pk), torch.bfloat16
    cfg, sets = L.LLaMAConfig(), 8
    with L.device_init(0.02):
        mlps = [L.MLPBF16(cfg) for _ in range(sets)]
        ats = [L.GroupedQueryAttentionBF16(cfg) for _ in range(sets)]
    h = torch.randn((B, WIDTH), device="cuda").to(bf)
    w = torch.ones(WIDTH, device="cuda", dtype=bf)
    K.hbm("add_rmsnorm_bf16", timed_graph(lambda i: ops.add_rmsnorm_bf16(h, h, w)), B * WIDTH * 8)
    K.hbm("product o", timed_graph(lambda i: ops.linear_bf16(h, ats[i % sets].o_proj)), WIDTH * WIDTH * 2 + B * WIDTH * 4)
    K.hbm("product k", timed_graph(lambda i: ops.linear_bf16(h, ats[i % sets].k_proj)), 256 * WIDTH * 2 + B * (WIDTH + 256) * 2)
    K.hbm("mlp (gate/up, down)", timed_graph(lambda i: mlps[i % sets](h, few_rows=True)), 3 * WIDTH * FF * 2 + B * WIDTH * 4)
    return K.out


def whole_models(B, S, window, n_blocks, steps):
    """Prompt pass and decode step of a Soluzen model and of a LLaMA model with as many layer runs, same width and batch."""
    from baranet_bdml_b200 import layers as L
    from baranet_bdml_b200.model import LLaMAModelBF16
    out = {}
    ids = torch.randint(0, VOCAB, (B, S), device="cuda", dtype=torch.int32)

    def one(model, runs):
        def prompt(i):
            model.prefill(ids, S + steps + 8)
        ms = timed(prompt, steps=3, warmup=2)
        tok = model.argmax(model.prefill(ids, S + steps + 8))
        step = model.capture_decode_step()
        dec = timed(lambda i: step(tok), steps=steps, warmup=3)
        model.status()
        r = {"layer_runs": runs, "parameters": sum(int(t.numel()) for t in model.parameters()), "prompt_ms": ms,
             "prompt_tokens_per_s": B * S / ms * 1e3, "decode_ms_per_step": dec, "decode_tokens_per_s": B / dec * 1e3}
        return r
    model = build(window, n_blocks)
    runs = len(model.runs)
    out["soluzen"] = one(model, runs)
    del model
    torch.cuda.empty_cache()
    cfg = L.LLaMAConfig(num_hidden_layers=runs, rms_norm_eps=1e-5)
    with L.device_init(0.02):
        model = LLaMAModelBF16(cfg)
    out["llama"] = one(model, runs)
    del model
    torch.cuda.empty_cache()
    out["config"] = {"batch": B, "prompt": S, "window": window, "width": WIDTH, "ff": FF, "vocab": VOCAB}
    return out


def run(pk, steps):
    torch.manual_seed(0)
    res = {"metric": "soluzen_throughput", "dtype": "bf16", "data": "synthetic", "peaks": pk, "l2": "inputs larger than L2, or rotated"}
    res["models"] = [whole_models(8, 2048, 1024, 2, steps), whole_models(16, 512, 1024, 2, steps), whole_models(64, 512, 4096, 1, steps)]
    res["prompt_kernels_16384_tokens"] = prompt_kernels(pk)
    torch.cuda.empty_cache()
    for B in (16, 64):
        res[f"step_kernels_{B}_rows"] = step_kernels(pk, B)
        torch.cuda.empty_cache()
    res["llama_step_kernels_16_rows"] = llama_step_kernels(pk, 16)
    return res
