"""Throughput of the Duponex design at sizes that resemble a real model's layers, beside the LLaMA family at equal width, heads
and parameters per layer: `python bench.py --duponex`.

Whole models (prompt pass, decode steps replayed from a CUDA graph) and every kernel of the design by itself, each against
its roofline, with the like kernel of the LLaMA family timed in the same run.  A kernel is timed with CUDA events over a loop
whose inputs together exceed the L2 (several sets of buffers where one set would fit)."""
from __future__ import annotations

import torch

from bench_soluzen import Kernels, RandomWeights, llama_step_kernels, timed, timed_graph

WIDTH, VOCAB, STREAMS = 2048, 32000, 2
HEADS, KV_HEADS, DIM = 32, 4, 64
FF = 7424                      # with the gate projection: as many parameters per layer as LLaMA at ff 5632


def attention(chunk, heads=HEADS, kv_heads=KV_HEADS, dim=DIM):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, mask={"size": chunk}, scale=dim ** -0.5, v_mix=True)


def config(chunk, n_layers, streams=STREAMS, **kw):
    layer = {"type": "attention", "mixer": attention(chunk, **kw), "mlp": {"kind": "dense", "ff": FF}}
    return {"architecture": "Duponex", "embedding": {"scale": 1.0}, "layers": [layer] * n_layers, "norm": {"eps": 1e-5},
            "residual_mult": 0.7, "streams": streams, "vocab": VOCAB, "width": WIDTH}


def weights():
    w = RandomWeights()

    def get(name, *shape):
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("ls1", "ls2", "in", "out", "vmix"):
            return torch.full(shape, 0.5, device="cuda", dtype=torch.bfloat16)
        if leaf == "mix" and len(shape) == 2:
            return torch.eye(shape[0], device="cuda", dtype=torch.bfloat16)
        return w(name, *shape)
    get.leftover = w.leftover
    return get


def build(chunk, n_layers, **kw):
    from baranet_bdml_b200 import _lib
    from baranet_bdml_b200.duponex import DuponexConfig, DuponexModel
    _lib.load()
    return DuponexModel(DuponexConfig.from_dict(config(chunk, n_layers, **kw)), weights())


def _mixer(chunk, **kw):
    from baranet_bdml_b200.mixers import ChunkedAttention, ChunkedAttentionConfig
    a = attention(chunk, **kw)
    cfg = ChunkedAttentionConfig(a["heads"], a["kv_heads"], a["dim"], a["vdim"], chunk, a["scale"], True)
    return ChunkedAttention(cfg, WIDTH, 1e-5, weights(), torch.bfloat16)


def _rnd(*shape, dtype=torch.bfloat16):
    return torch.randn(shape, device="cuda").to(dtype)


def _stream():
    return torch.cuda.current_stream().cuda_stream


def prompt_kernels(pk, B=8, S=2048):
    from baranet_bdml_b200 import _lib, ops
    from baranet_bdml_b200.mixers import MLP
    lib, K, bf, T = _lib.load(), Kernels(pk), torch.bfloat16, B * S
    seq, zero = torch.arange(B, dtype=torch.int32, device="cuda"), torch.zeros(B, dtype=torch.int32, device="cuda")
    h = _rnd(T, WIDTH)
    for dim, heads, kv in ((64, 32, 4), (128, 16, 4)):
        for chunk in (512, 2048):
            m = _mixer(chunk, dim=dim, heads=heads, kv_heads=kv)
            c, cache = m.cfg, m.new_state(B)
            proj = m.project(h)
            q, k, v, g = m._columns(proj)
            keys, vals, out, vf = _rnd(T, kv * dim), _rnd(T, kv * dim), _rnd(T, heads * dim), _rnd(T, kv * dim)
            seen = sum(i % chunk + 1 for i in range(S))

            def attn(i):
                _lib.check(lib.bn_attn_chunked(q, proj.stride(0), keys.data_ptr(), keys.stride(0), vals.data_ptr(), vals.stride(0), g,
                                               proj.stride(0), out.data_ptr(), out.stride(0), B, S, 0, S, heads, kv, dim, dim, chunk, dim, 1e-5,
                                               float(c.scale), m.score_bound, ops.status_word("cuda").data_ptr(), 1, _stream()))
            K.tensor(f"portion attention, {heads} x {dim}, chunk {chunk}", timed(attn), 2.0 * B * heads * seen * 2 * dim)

            def prep(i):
                _lib.check(lib.bn_kv_prep(k, v, proj.stride(0), vf.data_ptr(), vf.stride(0), 0.5, seq.data_ptr(), zero.data_ptr(), B, S, kv, dim,
                                          dim, dim, 1e-5, keys.data_ptr(), vals.data_ptr(), S, 0, cache.k.data_ptr(), cache.v.data_ptr(),
                                          cache.ring_tokens, chunk, 1, _stream()))
            kept = B * ((S - 1) % chunk + 1)
            K.hbm(f"kv_prep, {kv} x {dim}, chunk {chunk}", timed_graph(prep), (T * 5 + kept * 2) * kv * dim * 2)
            pos = torch.full((B,), chunk - 1, dtype=torch.int32, device="cuda")
            K.hbm(f"kv_gather, {kv} x {dim}, {chunk - 1} tokens", timed_graph(lambda i: cache.gather(seq, pos, chunk - 1, keys, vals, chunk - 1)),
                  B * (chunk - 1) * kv * dim * 8)
            if chunk == 512:
                K.tensor(f"product q|k|v|gate, {heads} x {dim}", timed(lambda i: m.project(h)), 2.0 * T * m.proj.n * m.proj.k)
                K.tensor(f"product o, {heads} x {dim}", timed(lambda i: m.o(out)), 2.0 * T * m.o.n * m.o.k)
    mlp = MLP(FF, WIDTH, "relu2", weights(), bf)
    u = mlp.up(h)
    K.tensor("product up with squared ReLU", timed(lambda i: mlp.up(h)), 2.0 * T * FF * WIDTH)
    K.tensor("product down", timed(lambda i: mlp.down(u)), 2.0 * T * FF * WIDTH)
    norm, scale = ops.NormWeight(torch.ones(WIDTH), None, 1e-5), torch.ones(WIDTH, device="cuda")
    for n in (2, 4):
        x = torch.randn((T, n, WIDTH), device="cuda")
        eye = [[float(i == j) for j in range(n)] for i in range(n)]
        for name, step, nbytes in ((f"hyper_norm {n} -> {n} streams", ops.StreamMix(eye, [0.5] * n, [0.5] * n), 8 * n + 4),
                                   (f"hyper_norm {n} -> sum", ops.StreamMix(eye, [0.5] * n, [1.0] * n, keep=False), 4 * n + 4)):
            K.hbm(name, timed(lambda i: ops.hyper_norm(x, step, bf, norm, delta=h, delta_scale=scale)), T * WIDTH * nbytes)
    ids = torch.randint(0, VOCAB, (T,), device="cuda", dtype=torch.int32)
    table, x = _rnd(VOCAB, WIDTH), torch.empty((T, WIDTH), device="cuda")
    K.hbm("embedding rows", timed(lambda i: ops.embedding_rows(table, ids, out_f32=x)), T * WIDTH * 6)
    return K.out


def llama_prompt_kernels(pk, B=8, S=2048):
    from baranet_bdml_b200 import ops
    K, bf, T = Kernels(pk), torch.bfloat16, B * S
    for b, s in ((B, S), (T // 512, 512)):
        q, k, v = _rnd(b, s, HEADS, DIM), _rnd(b, s, KV_HEADS, DIM), _rnd(b, s, KV_HEADS, DIM)
        ws = ops.prefill_workspace(b, s, HEADS, KV_HEADS, DIM)
        out = torch.empty_like(q)
        ops.attn_prefill_bf16(q, k, v, out=out, workspace=ws)
        K.tensor(f"prefill_kernel, causal, {b} x {s}",
                 timed(lambda i: ops.attn_prefill_bf16(q, None, v, out=out, workspace=ws, reuse_rotated_k=True)),
                 2.0 * b * HEADS * (s * (s + 1) / 2) * 2 * DIM)
    h, w = _rnd(T, WIDTH), torch.ones(WIDTH, device="cuda", dtype=bf)
    for name, n, kk in (("product 2048 x 2048", 2048, 2048), ("product 5120 x 2048", 5120, 2048), (f"product {FF} x 2048", FF, 2048),
                        (f"product 2048 x {FF}", 2048, FF)):
        x, wt = _rnd(T, kk), _rnd(n, kk)
        K.tensor(name, timed(lambda i: ops.gemm_bf16_nt(x, wt)), 2.0 * T * n * kk)
    K.hbm("add_rmsnorm_bf16", timed(lambda i: ops.add_rmsnorm_bf16(h, h, w)), T * WIDTH * 8)
    return K.out


def step_kernels(pk, B, chunk=4096, sets=8):
    from baranet_bdml_b200 import _lib, ops
    from baranet_bdml_b200.mixers import MLP
    lib, K, bf = _lib.load(), Kernels(pk), torch.bfloat16
    seq = torch.arange(B, dtype=torch.int32, device="cuda")
    h = _rnd(B, WIDTH)
    for dim, heads, kv in ((64, 32, 4), (128, 16, 4)):
        ms = [_mixer(chunk, dim=dim, heads=heads, kv_heads=kv) for _ in range(sets)]
        m = ms[0]
        caches = [m.new_state(B) for _ in range(sets)]
        for c in caches:
            c.k.normal_()
            c.v.normal_()
        proj = m.project(h)
        splits = lib.bn_gqa_step_splits(B, heads, kv, dim, dim, chunk, 1)
        for seen in (chunk, chunk // 2):
            pos = torch.full((B,), 3 * chunk + seen - 1, dtype=torch.int32, device="cuda")
            name = f"gqa_step, {heads} x {dim} over {kv}, {seen} of {chunk} keys"

            def attend(i):
                out = torch.empty((B, m.o.k), dtype=bf, device="cuda")
                m._one_token(proj, B, 1, caches[i % sets], seq, pos, None, m.values(proj), out)
            K.hbm(name, timed_graph(attend), B * seen * kv * dim * 4 + B * (m.proj.n + heads * dim) * 2)
            K.out[name]["splits"] = splits
        del caches

        def weight_stream(name, fn, lin):
            K.hbm(name, timed_graph(fn), lin.n * lin.k * 2 + B * (lin.n + lin.k) * 2)
        out = _rnd(B, m.o.k)
        weight_stream(f"product q|k|v|gate, {heads} x {dim}", lambda i: ms[i % sets].project(h), m.proj)
        weight_stream(f"product o, {heads} x {dim}", lambda i: ms[i % sets].o(out), m.o)
    mlps = [MLP(FF, WIDTH, "relu2", weights(), bf) for _ in range(sets)]
    u = _rnd(B, FF)
    weight_stream("product up with squared ReLU", lambda i: mlps[i % sets].up(h), mlps[0].up)
    weight_stream("product down", lambda i: mlps[i % sets].down(u), mlps[0].down)
    norm, scale = ops.NormWeight(torch.ones(WIDTH), None, 1e-5), torch.ones(WIDTH, device="cuda")
    for n in (2, 4):
        x = torch.randn((B, n, WIDTH), device="cuda")
        step = ops.StreamMix([[1.0] * n] * n, [0.5] * n, [0.5] * n)
        K.hbm(f"hyper_norm {n} -> {n} streams", timed_graph(lambda i: ops.hyper_norm(x, step, bf, norm, delta=h, delta_scale=scale)),
              B * WIDTH * (8 * n + 4))
    return K.out


def llama_decode_kernels(pk, B, seen=4096, sets=8):
    from baranet_bdml_b200.kv_cache import PAGE_TOKENS, PagedKVCache
    K = Kernels(pk)
    pages = seen // PAGE_TOKENS
    caches = []
    for _ in range(sets):
        c = PagedKVCache(B * pages, B, pages, KV_HEADS, DIM)
        c.pool.normal_()
        c.page_table.copy_(torch.arange(B * pages, dtype=torch.int32, device="cuda").view(B, pages))
        c.seq_lens.fill_(seen)
        caches.append(c)
    q = _rnd(B, HEADS, DIM)
    K.hbm(f"decode_paged_kernel, {seen} keys", timed_graph(lambda i: caches[i % sets].decode(q, num_heads=HEADS)), B * seen * KV_HEADS * DIM * 4)
    return K.out


def whole_models(B, S, chunk, n_layers, steps, streams=STREAMS):
    """Prompt pass and decode step of a Duponex model and of a LLaMA model with as many layers, same width, heads and batch."""
    from baranet_bdml_b200 import layers as L
    from baranet_bdml_b200.model import LLaMAModelBF16
    out = {}
    ids = torch.randint(0, VOCAB, (B, S), device="cuda", dtype=torch.int32)

    def one(model):
        room = S + 2 * steps + 16
        ms = timed(lambda i: model.prefill(ids, room), steps=3, warmup=2)
        tok = model.argmax(model.prefill(ids, room))
        step = model.capture_decode_step()
        dec = timed(lambda i: step(tok), steps=steps, warmup=3)
        model.status()
        return {"layers": n_layers, "parameters": sum(int(t.numel()) for t in model.parameters()), "prompt_ms": ms,
                "prompt_tokens_per_s": B * S / ms * 1e3, "decode_ms_per_step": dec, "decode_tokens_per_s": B / dec * 1e3}
    model = build(chunk, n_layers, streams=streams)
    out["duponex"] = one(model)
    del model
    torch.cuda.empty_cache()
    with L.device_init(0.02):
        model = LLaMAModelBF16(L.LLaMAConfig(num_hidden_layers=n_layers, rms_norm_eps=1e-5))
    out["llama"] = one(model)
    del model
    torch.cuda.empty_cache()
    out["config"] = {"batch": B, "prompt": S, "chunk": chunk, "streams": streams, "width": WIDTH, "ff": FF, "vocab": VOCAB}
    return out


def run(pk, steps):
    torch.manual_seed(0)
    res = {"metric": "duponex_throughput", "dtype": "bf16", "data": "synthetic", "peaks": pk, "l2": "inputs larger than L2, or rotated"}
    res["models"] = [whole_models(8, 2048, 1024, 12, steps), whole_models(8, 2048, 4096, 12, steps, streams=4),
                     whole_models(16, 512, 1024, 12, steps), whole_models(64, 512, 4096, 6, steps)]
    res["prompt_kernels_16384_tokens"] = prompt_kernels(pk)
    res["llama_prompt_kernels_16384_tokens"] = llama_prompt_kernels(pk)
    torch.cuda.empty_cache()
    for B in (16, 64):
        res[f"step_kernels_{B}_rows"] = step_kernels(pk, B)
        torch.cuda.empty_cache()
        res[f"llama_decode_{B}_rows"] = llama_decode_kernels(pk, B)
        torch.cuda.empty_cache()
    res["llama_step_kernels_16_rows"] = llama_step_kernels(pk, 16)
    return res
