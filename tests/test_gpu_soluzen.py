"""Soluzen on the GPU against the plain fp64 restatement (oracle/ref_soluzen.py): every mechanism alone, whole prompts,
portions, one-token steps, slots used again, and generation through the framework's entry point.

fp32 gate 1e-4, bf16 gate 5e-2, both of the root mean square of the expected rows.  A random model amplifies rounding at a
few positions (rounding the restatement's own activations to bf16 moves single rows by up to 0.2), so whole models in bf16
are held to the gate at nine rows in ten and to ten times the gate at every row; a single mechanism, and everything in
fp32, is held to its gate at every row.  `test_the_gates_see_planted_mistakes` plants mistakes in the restatement and
checks that they exceed the fp32 gate by far."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import soluzen_cases as K
from oracle import ref_soluzen as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GATE = {torch.float32: 1e-4, torch.bfloat16: 5e-2}
DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])


def assert_close(got, want, dtype, what=None):
    e = K.row_errors(got, want)
    if dtype == torch.float32:
        assert e.max() <= GATE[dtype], (what, e.max())
    else:
        assert np.quantile(e, 0.9) <= GATE[dtype] and e.max() <= 10 * GATE[dtype], (what, np.quantile(e, 0.9), e.max())


def make(name, dtype, seed=0):
    from baranet_bdml_b200 import registry
    from baranet_bdml_b200.checkpoint import Weights
    w = K.weights(K.CASES[name], seed)
    return registry.build_model(K.CASES[name], Weights(w), dtype), w


def tokens(name, n, seed=5):
    return np.random.default_rng(seed).integers(0, K.CASES[name]["vocab"], n).astype(np.int32)


def gpu(x, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(x, dtype=np.float32)).cuda().to(dtype)


def run_portions(model, slot, toks, sizes):
    """All logits of one sequence fed in portions of the given sizes (the last one repeats until the end)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        k += 1
        ids = torch.from_numpy(toks[at:at + n]).cuda()[None]
        out.append(model.extend(ids, [slot], torch.arange(n, device="cuda")).cpu())
        at += n
    model.status()
    return torch.cat(out).numpy()


# ------------------------------------------------------------------------------------------ whole models
@DTYPES
@pytest.mark.parametrize("name,n", [("odd", 61), ("even", 200), ("plain", 20), ("tail", 45)])
def test_whole_prompt_portions_and_steps(lib, name, n, dtype):
    model, w = make(name, dtype)
    toks = tokens(name, n)
    want = R.forward(K.CASES[name], K.as_f64(w), toks)
    model.allocate(2)
    for sizes in ([n], [1], [2], [3, 1, 7, 2, 16], [n // 2, 1, 1, 5], [n - 8, 1]):
        slot = model.slots.acquire()
        got = run_portions(model, slot, toks, sizes)
        assert_close(got, want, dtype, sizes)
        assert int(model.seq_lens[slot]) == n
        model.slots.release(slot)                      # the next schedule runs in a slot that has been used


@DTYPES
def test_layers_one_by_one(lib, dtype):
    """The residual stream after every layer run, through a model that is cut short behind that run."""
    from baranet_bdml_b200.ops import residual_norm
    model, w = make("odd", dtype)
    toks = tokens("odd", 33)
    after = []
    R.forward(K.CASES["odd"], K.as_f64(w), toks, after)
    runs = model.runs
    for k in range(1, len(runs) + 1):
        model.runs = runs[:k]
        model.allocate(1)
        slot = model.slots.acquire()
        ids, pos = torch.from_numpy(toks).cuda(), torch.zeros(1, dtype=torch.int32, device="cuda")
        x, pending = model._forward(ids, 1, len(toks), torch.tensor([slot], dtype=torch.int32, device="cuda"), pos, 0)
        x, _ = residual_norm(x, pending, dtype, model.config.width)
        assert_close(x.cpu().numpy(), after[k - 1], dtype, k)


@DTYPES
def test_long_decoding_past_every_window(lib, dtype):
    """150 tokens one by one behind a short prompt: the windows (7, 19) wrap their rings many times."""
    model, w = make("odd", dtype, seed=3)
    toks = tokens("odd", 160, 8)
    want = R.forward(K.CASES["odd"], K.as_f64(w), toks)
    model.allocate(1)
    got = run_portions(model, model.slots.acquire(), toks, [10, 1])
    assert_close(got, want, dtype)


@DTYPES
def test_unequal_sequences_step_together(lib, dtype):
    """Sequences of different lengths in one decode batch (also more rows than the weight-streaming kernels take) give what
    each gives alone."""
    name = "even"
    model, w = make(name, dtype, seed=2)
    lens = [3, 90, 17, 71, 1, 34, 69, 70, 64, 65, 2, 5, 8, 40, 33, 12, 9, 21]
    seqs = [tokens(name, n + 4, 100 + i) for i, n in enumerate(lens)]
    model.allocate(len(lens))
    slots = [model.slots.acquire() for _ in lens]
    for s, n, toks in zip(slots, lens, seqs):
        model.extend(torch.from_numpy(toks[:n]).cuda()[None], [s])
    got = [model.decode_step(torch.tensor([q[n + t] for q, n in zip(seqs, lens)], dtype=torch.int32, device="cuda")).cpu().numpy()
           for t in range(4)]
    want = [R.forward(K.CASES[name], K.as_f64(w), toks)[n:n + 4] for n, toks in zip(lens, seqs)]
    assert_close(np.stack(got, axis=1).reshape(4 * len(lens), -1), np.concatenate(want), dtype)
    # a step of some of them, in another order
    pick = [5, 0, 9]
    more = tokens(name, 3, 77)
    logits = model.decode_step(torch.from_numpy(more).cuda(), slots=[slots[i] for i in pick]).cpu().numpy()
    for r, i in enumerate(pick):
        want = R.forward(K.CASES[name], K.as_f64(w), np.concatenate([seqs[i], more[r:r + 1]]))
        assert K.error(logits[r:r + 1], want[-1:]) <= (GATE[dtype] if dtype == torch.float32 else 5 * GATE[dtype])


@DTYPES
def test_portions_of_several_sequences_together(lib, dtype):
    name = "even"
    model, w = make(name, dtype)
    seqs = np.stack([tokens(name, 110, s) for s in (1, 2, 3)])
    model.allocate(4)
    slots = [model.slots.acquire() for _ in range(4)][1:]
    got, at = [], 0
    for n in (40, 1, 45, 24):
        ids = torch.from_numpy(seqs[:, at:at + n].copy()).cuda()
        got.append(model.extend(ids, slots, torch.arange(3 * n, device="cuda")).cpu().numpy().reshape(3, n, -1))
        at += n
    got = np.concatenate(got, axis=1)
    for i in range(3):
        assert_close(got[i], R.forward(K.CASES[name], K.as_f64(w), seqs[i]), dtype, i)


def test_generate_greedy(lib):
    """generate() over prompts of unequal lengths picks, token by token, what the restatement picks wherever its best two
    logits are not closer than the fp32 gate; ids outside the vocabulary raise."""
    model, w = make("odd", torch.float32, seed=4)
    prompts = [list(map(int, tokens("odd", n, n))) for n in (5, 12, 1)]
    out = model.generate(prompts, max_new_tokens=9)
    for p, o in zip(prompts, out):
        assert o[:len(p)] == p and len(o) == len(p) + 9
        for k in range(len(p), len(o)):
            logits = R.forward(K.CASES["odd"], K.as_f64(w), o[:k])[-1]
            assert logits[o[k]] >= logits.max() - 1e-3
    assert model.generate(np.array([prompts[0]]), 9)[0] == out[0]
    with pytest.raises(IndexError):
        model.prefill([[1, K.CASES["odd"]["vocab"]]], 4)


def test_graphed_steps_equal_eager_ones(lib):
    toks = tokens("even", 6, 3)
    prompt = torch.from_numpy(tokens("even", 75, 9)).cuda()[None].repeat(2, 1)
    eager, _ = make("even", torch.bfloat16)
    eager.prefill(prompt, 100)
    want = [eager.decode_step(torch.tensor([t, t + 1], dtype=torch.int32, device="cuda")).clone() for t in toks]
    graphed, _ = make("even", torch.bfloat16)
    graphed.prefill(prompt, 100)
    step = graphed.capture_decode_step()
    for t, v in zip(toks, want):
        logits, nxt = step(torch.tensor([t, t + 1], dtype=torch.int32, device="cuda"))
        torch.cuda.synchronize()
        assert torch.equal(logits, v) and torch.equal(nxt, graphed.argmax(v))


def test_trace_and_command_line(lib, tmp_path):
    from baranet_bdml_b200.checkpoint import write_safetensors
    name = "tail"
    w = K.weights(K.CASES[name], 6)
    (tmp_path / "config.json").write_text(json.dumps(K.CASES[name]))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    toks = tokens(name, 30)
    want = R.forward(K.CASES[name], K.as_f64(w), toks)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:20].tolist(), "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[20:22].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[22:23].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks.tolist(), "want": [29]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (tmp_path / "1.f32").exists()
    for s, rows in ((0, [0, 19]), (2, [22]), (3, [29])):
        got = np.fromfile(tmp_path / f"{s}.f32", dtype="<f4").reshape(len(rows), -1)
        assert K.error(got, want[rows]) <= GATE[torch.float32]
    r = subprocess.run([sys.executable, "-m", "baranet_bdml_b200", "generate", "--model", str(tmp_path), "--dtype", "float32",
                        "--max-new-tokens", "3", "--prompt", "1 2 3", "--prompt", "4,5"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [len(line.split()) for line in r.stdout.splitlines()] == [6, 5]


def test_the_gates_see_planted_mistakes(lib):
    """Mistakes planted in the restatement move its logits by far more than the gates allow, so the tests above would see
    them in the product."""
    name, n = "odd", 61
    cfg, W, toks = K.CASES[name], K.as_f64(K.weights(K.CASES[name], 0)), tokens("odd", 61)
    want = R.forward(cfg, W, toks)

    def mistaken(change):
        c = json.loads(json.dumps(cfg))
        V = dict(W)
        change(c, V)
        return K.error(R.forward(c, V, toks), want)
    assert mistaken(lambda c, V: c["layers"][1]["mixer"]["mask"].update(size=8)) > 0.1
    assert mistaken(lambda c, V: c["layers"][3]["mixer"]["mask"].update(size=18)) > 0.1
    assert mistaken(lambda c, V: c["layers"][3]["mixer"]["rot"].update(base=520.0)) > 5e-4
    assert mistaken(lambda c, V: V.update({"loop.step": V["loop.step"][::-1]})) > 0.1
    assert mistaken(lambda c, V: V.update({"l2.mix.D": V["l2.mix.D"] * 1.2})) > 5e-2
    assert mistaken(lambda c, V: c["layers"][0]["mixer"].update(norm_groups=1)) > 5e-2


# ------------------------------------------------------------------------------------------ mechanisms alone
@DTYPES
@pytest.mark.parametrize("hidden", [72, 74, 2048, 5000])
def test_residual_norm(lib, dtype, hidden):
    from baranet_bdml_b200 import ops
    rng = np.random.default_rng(0)
    rows, w8 = 37, ops.round8(hidden)
    x, d = rng.standard_normal((rows, hidden)) * 3 + 1, rng.standard_normal((rows, hidden))
    row, wn, bn, dw = (rng.standard_normal(hidden) for _ in range(4))
    dg = torch.zeros((rows, w8), dtype=dtype, device="cuda")
    dg[:, :hidden] = gpu(d, dtype)
    d16 = dg[:, :hidden].double().cpu().numpy()
    f = lambda v: np.asarray(v, dtype=np.float32).astype(np.float64)          # noqa: E731
    x, row, wn, bn, dw = map(f, (x, row, wn, bn, dw))
    for own, r, b in ((None, None, bn), (dw, None, None), (dw, row, bn), (None, row, None)):
        cast = torch.zeros((rows, 2 * w8), dtype=dtype, device="cuda")
        p = ops.Pending(dg, None if own is None else ops.NormWeight(gpu(own), None, 1e-3))
        total, y = ops.residual_norm(gpu(x), p, dtype, hidden, row=None if r is None else gpu(r), cast=cast, lo_offset=w8,
                                     norm=ops.NormWeight(gpu(wn), None if b is None else gpu(b), 1e-2))
        want = x + (d16 if own is None else R.rms_norm(d16, own, 1e-3)) + (0 if r is None else r)
        assert np.abs(total.double().cpu().numpy() - want).max() <= 4e-6 * np.abs(want).max()
        wy = R.rms_norm(want, wn, 1e-2) if b is None else R.layer_norm(want, wn, b, 1e-2)
        tol = 1e-5 if dtype == torch.float32 else 2.0 ** -8
        assert np.abs(y[:, :hidden].double().cpu().numpy() - wy).max() <= tol * np.abs(wy).max()
        assert float(y[:, hidden:].float().abs().sum()) == 0
        both = cast[:, :hidden].double() + cast[:, w8:w8 + hidden].double()
        assert np.abs(both.cpu().numpy() - want).max() <= 2.0 ** -16 * np.abs(want).max()


def _linear_case(rows, n, k, dtype, seed=0):
    rng = np.random.default_rng(seed)
    x, w = gpu(rng.standard_normal((rows, k)), dtype), gpu(rng.standard_normal((n, k)) / np.sqrt(k), torch.bfloat16)
    return x, w, x.double().cpu().numpy() @ w.double().cpu().numpy().T


@DTYPES
@pytest.mark.parametrize("rows", [1, 7, 16, 40, 300])
@pytest.mark.parametrize("n,k", [(40, 52), (264, 320), (19, 12), (256, 512)])
def test_linear_forms(lib, dtype, rows, n, k):
    from baranet_bdml_b200 import ops
    x, w, want = _linear_case(rows, n, k, dtype)
    lin, n8 = ops.Linear(w, dtype), ops.round8(n)
    s = np.abs(want).max()
    tol = 2e-6 if dtype == torch.float32 else 2.0 ** -8
    y = lin(x)
    assert np.abs(y[:, :n].double().cpu().numpy() - want).max() <= tol * s and float(y[:, n:].float().abs().sum()) == 0
    y = lin(x, f32_out=True)
    assert y.dtype == torch.float32 and np.abs(y[:, :n].double().cpu().numpy() - want).max() <= 3e-6 * s
    # act(x W) * e, e a column range of a wider matrix
    rng = np.random.default_rng(1)
    wide = gpu(rng.standard_normal((rows, 3 * n8)), dtype)
    e = wide[:, n8:2 * n8]
    for act, f in (("gelu_tanh", R.gelu_tanh), ("silu", R.silu), ("none", lambda z: z)):
        ref = f(want) * e[:, :n].double().cpu().numpy()
        got = lin.act_mul(x, e, act)[:, :n].double().cpu().numpy()
        assert np.abs(got - ref).max() <= 2 * tol * np.abs(ref).max(), act
    x2, w2, up = _linear_case(rows, n, k, dtype)
    u = gpu(np.random.default_rng(9).standard_normal((n, k)) / np.sqrt(k), torch.bfloat16)
    upv = x.double().cpu().numpy() @ u.double().cpu().numpy().T
    for act, f in (("gelu_tanh", R.gelu_tanh), ("silu", R.silu)):
        ref = f(want) * upv
        got = ops.GatedLinear(w, u, act, dtype)(x)
        assert np.abs(got[:, :n].double().cpu().numpy() - ref).max() <= 2 * tol * np.abs(ref).max(), act
        assert float(got[:, n:].float().abs().sum()) == 0


def _window_attention(q, kn, kr, v, n_old, window, scale, dtype):
    """bn_attn_window on (T, H, .) arrays whose first n_old keys have no query; returns (T - n_old, H, V)."""
    from baranet_bdml_b200 import _lib, ops
    n, H, dim = kn.shape
    rot, vd, S = kr.shape[1], v.shape[2], n - n_old
    r8 = ops.round8
    qg = torch.zeros((S, r8(H * (dim + rot))), dtype=dtype, device="cuda")
    qg[:, :H * (dim + rot)] = gpu(q.reshape(S, -1), dtype)
    kv = torch.zeros((n, r8(H * (dim + vd))), dtype=dtype, device="cuda")
    kv[:, :H * dim], kv[:, H * dim:H * (dim + vd)] = gpu(kn.reshape(n, -1), dtype), gpu(v.reshape(n, -1), dtype)
    krg = torch.zeros((n, r8(rot)), dtype=dtype, device="cuda")
    krg[:, :rot] = gpu(kr, dtype)
    out = torch.full((S, r8(H * vd)), 7.0, dtype=dtype, device="cuda")
    word = torch.zeros(1, dtype=torch.int32, device="cuda")
    _lib.check(_lib.load().bn_attn_window(
        qg.data_ptr(), qg.stride(0), kv.data_ptr(), kv.data_ptr() + H * dim * kv.element_size(), kv.stride(0), krg.data_ptr(),
        krg.stride(0), out.data_ptr(), out.stride(0), 1, S, n_old, n, H, dim, rot, vd, window, scale, word.data_ptr(),
        0 if dtype == torch.float32 else 1, torch.cuda.current_stream().cuda_stream))
    torch.cuda.synchronize()
    assert int(word.item()) == 0
    up = lambda t: t.double().cpu().numpy()              # noqa: E731
    K_ = np.concatenate([up(kv[:, :H * dim]).reshape(n, H, dim), np.repeat(up(krg[:, :rot])[:, None], H, axis=1)], axis=2)
    Q_ = np.concatenate([np.zeros((n_old, H, dim + rot)), up(qg[:, :H * (dim + rot)]).reshape(S, H, dim + rot)])
    want = R.windowed_softmax_attention(Q_, K_, up(kv[:, H * dim:H * (dim + vd)]).reshape(n, H, vd), scale, window)[n_old:]
    return up(out[:, :H * vd]).reshape(S, H, vd), want


@DTYPES
@pytest.mark.parametrize("H,dim,rot,vd", [(2, 128, 64, 128), (3, 64, 32, 64), (2, 40, 16, 72), (1, 192, 64, 192), (2, 10, 6, 11), (2, 8, 8, 8)])
@pytest.mark.parametrize("S,n_old,window", [(300, 0, 1000), (129, 63, 64), (1, 40, 41), (2, 7, 3), (520, 199, 200), (260, 0, 1), (257, 126, 127),
                                            (256, 127, 128), (200, 128, 129)])
def test_window_attention(lib, dtype, H, dim, rot, vd, S, n_old, window):
    """Keys whose score stands out sit just inside and just outside every query's window: with q and k drawn so that a score
    reaches about 12, a key more or less changes the row outright."""
    rng = np.random.default_rng(S + window + dim)
    n = S + n_old
    q, kn = rng.standard_normal((S, H, dim + rot)), rng.standard_normal((n, H, dim))
    kr, v = rng.standard_normal((n, rot)), rng.standard_normal((n, H, vd))
    got, want = _window_attention(q, kn, kr, v, n_old, window, 4.0 * (dim + rot) ** -0.5, dtype)
    assert np.abs(got - want).max() <= (2e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("H,dim,rot,vd", [(20, 128, 64, 128), (32, 40, 16, 72), (16, 128, 64, 192)])
@pytest.mark.parametrize("S,window", [(70, 30), (130, 500), (300, 64)])
def test_window_attention_many_short_units(lib, H, dim, rot, vd, S, window):
    """More (sequence, head, query tile) units than the GPU has SMs, each of a few key tiles."""
    from baranet_bdml_b200 import _lib
    rng = np.random.default_rng(S + H)
    B, scale, bf = 12, 4.0 * (dim + rot) ** -0.5, torch.bfloat16
    q, kn = gpu(rng.standard_normal((B, S, H, dim + rot)), bf), gpu(rng.standard_normal((B, S, H, dim)), bf)
    kr, v = gpu(rng.standard_normal((B, S, rot)), bf), gpu(rng.standard_normal((B, S, H, vd)), bf)
    kv = torch.cat([kn.reshape(B * S, -1), v.reshape(B * S, -1)], dim=1).contiguous()
    out, word = torch.zeros((B, S, H, vd), dtype=bf, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    for _ in range(3):
        _lib.check(_lib.load().bn_attn_window(
            q.data_ptr(), H * (dim + rot), kv.data_ptr(), kv.data_ptr() + H * dim * 2, kv.stride(0), kr.data_ptr(), rot, out.data_ptr(), H * vd,
            B, S, 0, S, H, dim, rot, vd, window, scale, word.data_ptr(), 1, torch.cuda.current_stream().cuda_stream))
    torch.cuda.synchronize()
    assert int(word.item()) == 0
    up = lambda t: t.double().cpu().numpy()              # noqa: E731
    for b in (0, B - 1):
        for h in (0, H - 1):
            key = np.concatenate([up(kn[b, :, h]), up(kr[b])], axis=1)[:, None]
            want = R.windowed_softmax_attention(up(q[b, :, h])[:, None], key, up(v[b, :, h])[:, None], scale, window)[:, 0]
            assert np.abs(up(out[b, :, h]) - want).max() <= 3e-2


@pytest.mark.parametrize("S", [64, 300])
def test_window_attention_growing_scores(lib, S):
    """Scores that rise along the keys by far more than the rescale threshold, and rows whose first key tile they cannot see."""
    rng = np.random.default_rng(0)
    H, dim, rot, vd = 2, 64, 64, 64
    q = np.abs(rng.standard_normal((S, H, dim + rot)))
    kn = np.abs(rng.standard_normal((S, H, dim))) * np.linspace(0.1, 6.0, S)[:, None, None]
    kr, v = rng.standard_normal((S, rot)), rng.standard_normal((S, H, vd))
    for window in (S, 70):
        got, want = _window_attention(q, kn, kr, v, 0, window, 0.3, torch.bfloat16)
        assert np.abs(got - want).max() <= 3e-2


@DTYPES
@pytest.mark.parametrize("H,kr,rot,window", [(4, 64, 32, 50), (17, 256, 64, 130), (16, 512, 64, 200), (3, 36, 10, 7), (2, 104, 16, 64)])
def test_latent_decode_over_the_ring(lib, dtype, H, kr, rot, window):
    """One token per row against rings that are partly filled, full and wrapped, rows in slots of their own."""
    from baranet_bdml_b200 import _lib
    from baranet_bdml_b200.kv_cache import LatentRingCache
    rng = np.random.default_rng(H + window)
    positions = [0, 1, window - 2, window - 1, window, window + 5, 3 * window + 7, 63, 64, 65]
    B = len(positions)
    cache = LatentRingCache(B + 2, window, kr, rot, dtype)
    slots = rng.permutation(B + 2)[:B].astype(np.int32)
    lat = [rng.standard_normal((p + 1, kr + rot)) for p in positions]
    cache.ring.fill_(9.0)                                   # rows that no sequence has written must not be seen
    if cache.kv_ld > kr:
        cache.ring[:, :, kr:cache.kv_ld] = 0
    cache.ring[:, :, cache.kv_ld + rot:] = 0
    for s, p, x in zip(slots, positions, lat):
        for t in range(max(0, p + 1 - cache.ring_tokens), p + 1):
            row = cache.ring[int(s), t % cache.ring_tokens]
            row[:kr], row[cache.kv_ld:cache.kv_ld + rot] = gpu(x[t, :kr], dtype), gpu(x[t, kr:], dtype)
    q = rng.standard_normal((B, H, kr + rot))
    qg = torch.zeros((B, H, cache.kv_ld + cache.rot_ld), dtype=dtype, device="cuda")
    qg[:, :, :kr], qg[:, :, cache.kv_ld:cache.kv_ld + rot] = gpu(q[:, :, :kr], dtype), gpu(q[:, :, kr:], dtype)
    scale = 4.0 * (kr + rot) ** -0.5
    L = _lib.load()
    dt = 0 if dtype == torch.float32 else 1
    sl, ps = torch.from_numpy(slots).cuda(), torch.tensor(positions, dtype=torch.int32, device="cuda")
    for splits in {1, 2, 3, L.bn_latent_decode_splits(B, H, kr, rot, window, dt)}:
        part = torch.full((B, H, splits, cache.kv_ld), 5.0, device="cuda")
        lse = torch.full((B, H, splits), 5.0, device="cuda")
        _lib.check(L.bn_latent_decode(qg.data_ptr(), cache.ring.data_ptr(), B + 2, cache.ring_tokens, sl.data_ptr(), ps.data_ptr(),
                                      part.data_ptr(), lse.data_ptr(), splits, B, H, kr, rot, window, scale, dt,
                                      torch.cuda.current_stream().cuda_stream))
        torch.cuda.synchronize()
        pt, ls = part.double().cpu().numpy()[..., :kr], lse.double().cpu().numpy()
        wgt = np.exp(ls - ls.max(axis=2, keepdims=True))
        got = (pt * wgt[..., None]).sum(2) / wgt.sum(2)[..., None]
        for b, (p, x) in enumerate(zip(positions, lat)):
            x = gpu(x, dtype).double().cpu().numpy()[max(0, p - window + 1):]
            qb = gpu(q[b], dtype).double().cpu().numpy()
            s = qb @ x.T * scale
            w = np.exp(s - s.max(1, keepdims=True))
            want = (w / w.sum(1, keepdims=True)) @ x[:, :kr]
            assert np.abs(got[b] - want).max() <= (2e-5 if dtype == torch.float32 else 3e-2), (b, p, splits)


@DTYPES
@pytest.mark.parametrize("H,P,G,N", [(4, 64, 1, 128), (4, 32, 2, 64), (3, 48, 3, 32), (2, 80, 1, 16), (6, 20, 3, 12), (2, 24, 1, 40), (1, 8, 1, 200)])
def test_scan_carries_its_state(lib, dtype, H, P, G, N):
    """The recurrence in pieces of unequal length, from a state that is not zero, two sequences in slots of their own; some
    heads decay within a token, some hardly at all."""
    from baranet_bdml_b200 import _lib, ops
    rng = np.random.default_rng(N + P)
    S, B, inner = 150, 2, H * P
    C = inner + 2 * G * N
    ld = ops.round8(C)
    xbc = torch.zeros((B, S, ld), dtype=dtype, device="cuda")
    xbc[:, :, :C] = gpu(rng.standard_normal((B, S, C)), dtype)
    dt = gpu(np.logaddexp(0, rng.standard_normal((B, S, H))))
    A = gpu(-np.exp(np.linspace(-6.0, 2.0, H) if H > 1 else np.array([-3.0])))
    a, D = (dt * A).contiguous(), gpu(rng.standard_normal(H))
    state = gpu(rng.standard_normal((3, H, P, N)))
    start = state.double().cpu().numpy()
    slots = torch.tensor([2, 0], dtype=torch.int32, device="cuda")
    got = []
    for lo, hi in ((0, 1), (1, 3), (3, 67), (67, 68), (68, 150)):
        n = hi - lo
        y = torch.zeros((B, n, ops.round8(inner)), dtype=dtype, device="cuda")
        part, dp, ap = (t[:, lo:hi].contiguous() for t in (xbc, dt, a))
        _lib.check(_lib.load().bn_ssm_scan(part.data_ptr(), ld, dp.data_ptr(), ap.data_ptr(), D.data_ptr(), state.data_ptr(), slots.data_ptr(),
                                           B, n, H, P, G, N, y.data_ptr(), y.stride(1), 0 if dtype == torch.float32 else 1,
                                           torch.cuda.current_stream().cuda_stream))
        got.append(y[:, :, :inner].double().cpu().numpy())
    got = np.concatenate(got, axis=1).reshape(B, S, H, P)
    X = xbc[:, :, :C].double().cpu().numpy()
    dn, An, Dn = dt.double().cpu().numpy(), A.double().cpu().numpy(), D.double().cpu().numpy()
    grp = np.arange(H) // (H // G)
    tol_y, tol_s = (2e-5, 2e-5) if dtype == torch.float32 else (2.0 ** -8, 1e-4)
    for b, slot in enumerate((2, 0)):
        St = start[slot].copy()
        want = np.empty((S, H, P))
        for t in range(S):
            x, Bt, Ct = X[b, t, :inner].reshape(H, P), X[b, t, inner:inner + G * N].reshape(G, N)[grp], X[b, t, inner + G * N:].reshape(G, N)[grp]
            St = np.exp(An * dn[b, t])[:, None, None] * St + dn[b, t][:, None, None] * x[:, :, None] * Bt[:, None, :]
            want[t] = np.einsum("hpn,hn->hp", St, Ct) + Dn[:, None] * x
        assert np.abs(got[b] - want).max() <= tol_y * np.abs(want).max()
        assert np.abs(state[slot].double().cpu().numpy() - St).max() <= tol_s * np.abs(St).max()
    assert np.array_equal(state[1].double().cpu().numpy(), start[1])


@DTYPES
@pytest.mark.parametrize("sizes", [dict(), dict(heads=2, vdim=64, state=128, groups=1, conv=4, norm_groups=1),
                                   dict(heads=4, vdim=12, state=256, groups=2, conv=1, norm_groups=2),
                                   dict(heads=1, vdim=33, state=300, groups=1, conv=7, norm_groups=3)])
def test_mamba_mixer_alone(lib, dtype, sizes):
    from baranet_bdml_b200.mixers import Mamba2Mixer
    from baranet_bdml_b200.soluzen import _mixer_config
    cfg = K.config([K.layer(K.mamba(**sizes))], 56, 16, 8)
    _mixer_alone(cfg, Mamba2Mixer(_mixer_config("mamba2", cfg["layers"][0]["mixer"]), 56, 1e-5, _get(cfg), dtype), R.mamba2, dtype)


@DTYPES
@pytest.mark.parametrize("sizes", [dict(), dict(heads=2, dim=64, rot_dim=64, vdim=128, q_rank=32, kv_rank=128, window=64),
                                   dict(heads=1, dim=5, rot_dim=2, vdim=3, q_rank=1, kv_rank=4, window=2, base=3.0, scale=0.9)])
def test_latent_attention_alone(lib, dtype, sizes):
    from baranet_bdml_b200.mixers import LatentAttention
    from baranet_bdml_b200.soluzen import _mixer_config
    cfg = K.config([K.layer(K.attention(**sizes))], 56, 16, 8)
    _mixer_alone(cfg, LatentAttention(_mixer_config("latent_attention", cfg["layers"][0]["mixer"]), 56, 1e-5, _get(cfg), dtype),
                 R.latent_attention, dtype)


def _get(cfg):
    w = K.weights(cfg, 11)
    return lambda name, *shape: w["l0.mix." + name].reshape(shape if shape else w["l0.mix." + name].shape)


def _mixer_alone(cfg, mixer, restatement, dtype):
    """A mixer over rows of its own choosing, cut in several ways, two sequences with different inputs."""
    W = K.as_f64(K.weights(cfg, 11))
    T, B = 140, 2
    h = gpu(np.random.default_rng(12).standard_normal((B, T, 56)), dtype)
    want = np.stack([restatement(h[b].double().cpu().numpy(), lambda s: W["l0.mix." + s], cfg["layers"][0]["mixer"], 1e-5) for b in range(B)])
    seq = torch.tensor([1, 0], dtype=torch.int32, device="cuda")
    for sizes in ([T], [3, 1, 64, 2, 1, 69], [70] + [1] * 70, [1, 2] * 46 + [2]):
        st = mixer.new_state(2)
        got, at = [], 0
        for n in sizes:
            pos = torch.full((B,), at, dtype=torch.int32, device="cuda")
            y = mixer(h[:, at:at + n].reshape(B * n, 56).contiguous(), B, n, st, seq, pos, None if n == 1 else at)
            got.append(y[:, :56].double().cpu().numpy().reshape(B, n, 56))
            at += n
        assert at == T
        assert K.error(np.concatenate(got, axis=1), want) <= (1e-5 if dtype == torch.float32 else 3e-2), sizes[:6]


def test_llama_checkpoint_through_the_registry(lib):
    """The family that was there before loads and generates through the same registry."""
    from baranet_bdml_b200 import registry
    from baranet_bdml_b200.checkpoint import Weights
    cfg = {"architecture": "LLaMA", "vocab_size": 200, "hidden_size": 128, "intermediate_size": 256, "num_hidden_layers": 2,
           "num_attention_heads": 2, "num_key_value_heads": 1, "eos_token_id": 199}
    np.random.seed(0)
    model = registry.build_model(cfg, None)
    names = {"embed_tokens": model.embed_tokens, "norm": model.norm_weight, "lm_head": model.lm_head}
    for i, lay in enumerate(model.layers):
        for part, obj in (("self_attn", lay.self_attn), ("mlp", lay.mlp)):
            for n in ("q_proj", "k_proj", "v_proj", "o_proj") if part == "self_attn" else ("gate_proj", "up_proj", "down_proj"):
                names[f"layers.{i}.{part}.{n}"] = getattr(obj, n)
        names[f"layers.{i}.input_layernorm"] = lay.input_layernorm_weight
        names[f"layers.{i}.post_attention_layernorm"] = lay.post_attention_layernorm_weight
    np.random.seed(1)
    other = registry.build_model(cfg, Weights({k: v.cpu() for k, v in names.items()}))
    prompt = np.arange(3, 13, dtype=np.int32)[None]
    assert other.generate(prompt, 5) == model.generate(prompt, 5)
    with pytest.raises(ValueError):
        model.generate([[1, 2], [3]], 2)
    with pytest.raises(registry.UnsupportedDtype):
        registry.build_model(cfg, None, torch.float32)
