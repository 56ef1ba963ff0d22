"""Duponex on the GPU against the plain fp64 restatement (oracle/ref_duponex.py): every mechanism alone, whole prompts, portions,
one-token steps, slots used again, and generation through the framework's entry point.

fp32 gate 1e-4, bf16 gate 5e-2, both of the root mean square of the expected rows.  A random model amplifies rounding at a few
positions, so whole models in bf16 are held to the gate at nine rows in ten and to six times the gate at every row; a single
mechanism, and everything in fp32, is held to its gate at every row.  What mistakes would do to the logits is measured in
test_duponex_host.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import duponex_cases as K
from oracle import ref_duponex as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GATE = {torch.float32: 1e-4, torch.bfloat16: 5e-2}
DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])


def assert_close(got, want, dtype, what=None):
    e = K.row_errors(got, want)
    if dtype == torch.float32:
        assert e.max() <= GATE[dtype], (what, e.max())
    else:
        assert np.quantile(e, 0.9) <= GATE[dtype] and e.max() <= 6 * GATE[dtype], (what, np.quantile(e, 0.9), e.max())


def make(name, dtype, seed=0):
    from baranet_bdml_b200 import registry
    from baranet_bdml_b200.checkpoint import Weights
    w = K.weights(K.CASES[name], seed)
    return registry.build_model(K.CASES[name], Weights(w), dtype), w


def tokens(name, n, seed=5):
    return np.random.default_rng(seed).integers(0, K.CASES[name]["vocab"], n).astype(np.int32)


def gpu(x, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(x, dtype=np.float32)).cuda().to(dtype)


def f64(t):
    return t.double().cpu().numpy()


def ints(x):
    return torch.tensor(list(map(int, x)), dtype=torch.int32, device="cuda")


def stream():
    return torch.cuda.current_stream().cuda_stream


def code(dtype):
    return 0 if dtype == torch.float32 else 1


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
@pytest.mark.parametrize("name,n", [("odd", 61), ("even", 220), ("plain", 20), ("wide", 90)])
def test_whole_prompt_portions_and_steps(lib, name, n, dtype):
    model, w = make(name, dtype)
    toks = tokens(name, n)
    want = R.forward(K.CASES[name], K.as_f64(w), toks)
    for limit in (None, n):
        model.allocate(2, limit)
        for sizes in ([n], [1], [2], [3, 1, 7, 2, 16], [n // 2, 1, 1, 5], [n - 8, 1], [33, 37, 26, 1]):
            slot = model.slots.acquire()
            assert_close(run_portions(model, slot, toks, sizes), want, dtype, sizes)
            assert int(model.seq_lens[slot]) == n
            model.slots.release(slot)                      # the next schedule runs in a slot that has been used
    with pytest.raises(RuntimeError, match="allocated for"):
        run_portions(model, model.slots.acquire(), np.concatenate([toks, toks[:1]]), [n + 1])


@DTYPES
def test_layers_one_by_one(lib, dtype):
    """The sum of the streams after every layer, through a model that ends there."""
    from baranet_bdml_b200 import registry
    from baranet_bdml_b200.checkpoint import Weights
    cfg, toks, w = K.CASES["odd"], tokens("odd", 33), K.weights(K.CASES["odd"], 0)
    after = []
    R.forward(cfg, K.as_f64(w), toks, after)
    for k in range(1, len(cfg["layers"]) + 1):
        cut = dict(cfg, layers=cfg["layers"][:k])
        model = registry.build_model(cut, Weights({n: w[n] for n in K.shapes(cut)}), dtype)
        model.allocate(1)
        x, delta, scale = model._forward(torch.from_numpy(toks).cuda(), 1, len(toks), ints([model.slots.acquire()]), ints([0]), 0)
        step = model.steps[-1]                              # the streams' sum, before its norm
        got = np.einsum("s,rsw->rw", np.array(step.mix), f64(x)) + step.w_out[0] * f64(delta)[:, :cfg["width"]] * f64(scale)
        assert_close(got, after[k - 1], dtype, k)


@DTYPES
def test_long_decoding_through_many_chunks(lib, dtype):
    """150 tokens one by one behind a short prompt: chunks of 7, 19, 16 and 5 begin many times."""
    model, w = make("odd", dtype, seed=3)
    toks = tokens("odd", 160, 8)
    want = R.forward(K.CASES["odd"], K.as_f64(w), toks)
    model.allocate(1)
    assert_close(run_portions(model, model.slots.acquire(), toks, [10, 1]), want, dtype)


@DTYPES
def test_unequal_sequences_step_together(lib, dtype):
    """Sequences of different lengths in one decode batch (also more rows than the weight-streaming kernels take) give what
    each gives alone."""
    name = "even"
    model, w = make(name, dtype, seed=2)
    lens = [3, 90, 17, 71, 1, 32, 69, 70, 64, 65, 2, 5, 8, 40, 33, 12, 94, 21]
    seqs = [tokens(name, n + 4, 100 + i) for i, n in enumerate(lens)]
    model.allocate(len(lens))
    slots = [model.slots.acquire() for _ in lens]
    for s, n, toks in zip(slots, lens, seqs):
        model.extend(torch.from_numpy(toks[:n]).cuda()[None], [s])
    got = [model.decode_step(ints([q[n + t] for q, n in zip(seqs, lens)])).cpu().numpy() for t in range(4)]
    want = [R.forward(K.CASES[name], K.as_f64(w), toks)[n:n + 4] for n, toks in zip(lens, seqs)]
    assert_close(np.stack(got, axis=1).reshape(4 * len(lens), -1), np.concatenate(want), dtype)
    # a step of some of them, in another order
    pick = [5, 0, 9]
    more = tokens(name, 3, 77)
    logits = model.decode_step(torch.from_numpy(more).cuda(), slots=[slots[i] for i in pick]).cpu().numpy()
    for r, i in enumerate(pick):
        want = R.forward(K.CASES[name], K.as_f64(w), np.concatenate([seqs[i], more[r:r + 1]]))
        assert K.error(logits[r:r + 1], want[-1:]) <= (GATE[dtype] if dtype == torch.float32 else 4 * GATE[dtype])


@DTYPES
def test_portions_of_several_sequences_together(lib, dtype):
    name = "even"
    model, w = make(name, dtype)
    seqs = np.stack([tokens(name, 150, s) for s in (1, 2, 3)])
    model.allocate(4)
    slots = [model.slots.acquire() for _ in range(4)][1:]
    got, at = [], 0
    for n in (40, 1, 55, 30, 24):
        ids = torch.from_numpy(seqs[:, at:at + n].copy()).cuda()
        got.append(model.extend(ids, slots, torch.arange(3 * n, device="cuda")).cpu().numpy().reshape(3, n, -1))
        at += n
    got = np.concatenate(got, axis=1)
    for i in range(3):
        assert_close(got[i], R.forward(K.CASES[name], K.as_f64(w), seqs[i]), dtype, i)


def test_a_result_does_not_depend_on_the_cut(lib):
    """bf16 rows of one prompt, cut in different ways, differ by rounding only: by less than a third of what bf16 differs from
    the restatement at its worst."""
    model, w = make("even", torch.bfloat16, seed=7)
    toks = tokens("even", 200, 9)
    model.allocate(3)
    runs = [run_portions(model, model.slots.acquire(), toks, sizes) for sizes in ([200], [70, 26, 1, 33], [150, 1])]
    for r in runs[1:]:
        e = K.row_errors(r, runs[0])
        assert np.quantile(e, 0.9) <= 2e-2 and e.max() <= 0.1


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
    prompt = torch.from_numpy(tokens("even", 66, 9)).cuda()[None].repeat(2, 1)
    eager, _ = make("even", torch.bfloat16)
    eager.prefill(prompt, 100)
    want = [eager.decode_step(ints([t, t + 1])).clone() for t in toks]
    graphed, _ = make("even", torch.bfloat16)
    graphed.prefill(prompt, 100)
    step = graphed.capture_decode_step()
    for t, v in zip(toks, want):
        logits, nxt = step(ints([t, t + 1]))
        torch.cuda.synchronize()
        assert torch.equal(logits, v) and torch.equal(nxt, graphed.argmax(v))


def test_trace_and_command_line(lib, tmp_path):
    from baranet_bdml_b200.checkpoint import write_safetensors
    name = "wide"
    w = K.weights(K.CASES[name], 6)
    (tmp_path / "config.json").write_text(json.dumps(K.CASES[name]))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    toks = tokens(name, 70)
    want = R.forward(K.CASES[name], K.as_f64(w), toks)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:40].tolist(), "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[40:42].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[42:43].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks.tolist(), "want": [69]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "70"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (tmp_path / "1.f32").exists()
    for s, rows in ((0, [0, 39]), (2, [42]), (3, [69])):
        got = np.fromfile(tmp_path / f"{s}.f32", dtype="<f4").reshape(len(rows), -1)
        assert K.error(got, want[rows]) <= GATE[torch.float32]
    r = subprocess.run([sys.executable, "-m", "baranet_bdml_b200", "generate", "--model", str(tmp_path), "--dtype", "bfloat16",
                        "--max-new-tokens", "3", "--prompt", "1 2 3", "--prompt", "4,5"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [len(line.split()) for line in r.stdout.splitlines()] == [6, 5]


# ------------------------------------------------------------------------------------------ mechanisms alone
@DTYPES
@pytest.mark.parametrize("hidden", [72, 74, 2048, 4096, 5000])
@pytest.mark.parametrize("n_in,n_out,keep", [(1, 1, True), (1, 3, True), (2, 2, True), (3, 3, True), (4, 4, True), (4, 4, False), (2, 2, False),
                                             (5, 5, True), (2, 4, True), (16, 16, False)])
def test_hyper_norm(lib, dtype, hidden, n_in, n_out, keep):
    from baranet_bdml_b200 import ops
    rng = np.random.default_rng(hidden + n_in)
    rows, w8 = 19, ops.round8(hidden)
    f = lambda v: np.asarray(v, dtype=np.float32).astype(np.float64)          # noqa: E731
    x, wn, ls = f(rng.standard_normal((rows, n_in, hidden)) * 2 + 0.5), f(rng.standard_normal(hidden)), f(rng.standard_normal(hidden))
    mix, w_out, w_in = f(rng.standard_normal((n_in, n_out))), f(rng.standard_normal(n_out)), f(rng.standard_normal(n_out))
    dg = torch.full((rows, w8), 3.0, dtype=dtype, device="cuda")
    dg[:, :hidden] = gpu(rng.standard_normal((rows, hidden)), dtype)
    step = ops.StreamMix(mix.tolist(), w_out, w_in, keep=keep)
    for delta, scale in ((None, None), (dg, gpu(ls)), (dg, None)):
        new, y = ops.hyper_norm(gpu(x), step, dtype, ops.NormWeight(gpu(wn), None, 1e-2), delta=delta, delta_scale=scale)
        y2 = 0.0 if delta is None else f64(dg)[:, :hidden] * (1.0 if scale is None else ls)
        want = R.write_streams(x.transpose(1, 0, 2), mix, w_out, y2 + np.zeros((rows, hidden)))
        if keep:
            assert np.abs(f64(new).transpose(1, 0, 2) - want).max() <= 4e-6 * np.abs(want).max()
        else:
            assert new is None
        wy = R.rms_norm(R.read_streams(want, w_in), wn, 1e-2)
        assert np.abs(f64(y)[:, :hidden] - wy).max() <= (2e-5 if dtype == torch.float32 else 2.0 ** -8) * np.abs(wy).max()
        assert float(y[:, hidden:].float().abs().sum()) == 0


@DTYPES
@pytest.mark.parametrize("rows", [1, 7, 16, 40, 300])
@pytest.mark.parametrize("n,k", [(40, 52), (264, 320), (19, 12), (256, 512)])
def test_linear_with_bias_and_activation(lib, dtype, rows, n, k):
    from baranet_bdml_b200 import ops
    rng = np.random.default_rng(n + rows)
    x, w = gpu(rng.standard_normal((rows, k)), dtype), gpu(rng.standard_normal((n, k)) / np.sqrt(k), torch.bfloat16)
    b = gpu(rng.standard_normal(n), torch.bfloat16)
    z = f64(x) @ f64(w).T
    for bias in (None, b):
        for act, f in (("none", lambda v: v), ("relu2", R.squared_relu)):
            want = f(z + (0.0 if bias is None else f64(b)))
            y = ops.Linear(w, dtype, bias=bias, act=act)(x)
            assert np.abs(f64(y)[:, :n] - want).max() <= (4e-6 if dtype == torch.float32 else 2.0 ** -8) * np.abs(want).max(), (bias is None, act)
            assert float(y[:, n:].float().abs().sum()) == 0
    with pytest.raises(RuntimeError):
        ops.Linear(w, torch.bfloat16, bias=b)(x.to(torch.bfloat16), f32_out=True)


def _pad(x, dtype):
    """(..., heads, d) -> GPU (..., heads * round8(d)) rows with zeros behind each head"""
    from baranet_bdml_b200.ops import round8
    t = torch.zeros(x.shape[:-1] + (round8(x.shape[-1]),), dtype=dtype, device="cuda")
    t[..., :x.shape[-1]] = gpu(x, dtype)
    return t.reshape(x.shape[:-2] + (-1,))


def _unpad(t, heads, d):
    return f64(t).reshape(t.shape[:-1] + (heads, -1))[..., :d]


def _chunked_attention(q, k, v, gate, n_old, chunk, scale, eps, dtype, bound=0.0):
    """bn_attn_chunked on (T, heads, .) arrays whose first n_old keys have no query; queries as projected, keys prepared."""
    from baranet_bdml_b200 import _lib
    n, G, E = k.shape
    S, H, V = q.shape[0], q.shape[1], v.shape[2]
    qg, kg, vg, gg = (_pad(a, dtype) for a in (q, k, v, gate))
    out = torch.full((S, vg.shape[1] // G * H), 7.0, dtype=dtype, device="cuda")
    word = torch.zeros(1, dtype=torch.int32, device="cuda")
    _lib.check(_lib.load().bn_attn_chunked(
        qg.data_ptr(), qg.stride(0), kg.data_ptr(), kg.stride(0), vg.data_ptr(), vg.stride(0), gg.data_ptr(), gg.stride(0), out.data_ptr(),
        out.stride(0), 1, S, n_old, n, H, G, kg.shape[1] // G, vg.shape[1] // G, chunk, E, eps, scale, bound, word.data_ptr(), code(dtype),
        stream()))
    torch.cuda.synchronize()
    assert int(word.item()) == 0
    Q = np.concatenate([np.zeros((n_old, H, E)), R.unit_rms(_unpad(qg, H, E), eps)])
    want = R.chunked_attention(Q, _unpad(kg, G, E), _unpad(vg, G, V), scale, chunk)[n_old:] * R.sigmoid(_unpad(gg, H, V))
    return _unpad(out, H, V), want


@DTYPES
@pytest.mark.parametrize("H,G,E,V", [(4, 2, 64, 64), (2, 1, 128, 128), (3, 3, 40, 72), (6, 1, 10, 11), (2, 2, 192, 40), (4, 2, 48, 136)])
@pytest.mark.parametrize("S,n_old,chunk", [(300, 0, 1000), (129, 63, 64), (1, 40, 41), (2, 2, 3), (520, 199, 200), (260, 0, 1), (257, 126, 127),
                                           (256, 127, 128), (200, 128, 129), (450, 37, 300)])
def test_chunked_attention(lib, dtype, H, G, E, V, S, n_old, chunk):
    """Sharp scores, so that a key more or less at a chunk's edge changes the row outright."""
    rng = np.random.default_rng(S + chunk + E)
    n = S + n_old
    q, k = 3.0 * rng.standard_normal((S, H, E)) * rng.uniform(0.1, 2.0, (S, H, 1)), R.unit_rms(rng.standard_normal((n, G, E)), 1e-5)
    v, g, scale = rng.standard_normal((n, G, V)), 2 * rng.standard_normal((S, H, V)), 4.0 * E ** -0.5
    for bound in (0.0, 1.02 * E * scale):
        got, want = _chunked_attention(q, k, v, g, n_old, chunk, scale, 1e-5, dtype, bound)
        assert np.abs(got - want).max() <= (2e-5 if dtype == torch.float32 else 3e-2), bound


@DTYPES
@pytest.mark.parametrize("B,H,G,E,V", [(16, 32, 4, 64, 64), (9, 40, 8, 128, 128), (20, 16, 2, 40, 136)])
@pytest.mark.parametrize("S,n_old,chunk", [(40, 0, 16), (130, 0, 500), (2, 9, 12), (300, 63, 64), (257, 0, 1)])
def test_many_short_units(lib, dtype, B, H, G, E, V, S, n_old, chunk):
    """More (sequence, head, query tile) units than the GPU has SMs, each of one or a few key tiles: the persistent kernel goes
    from unit to unit while the one before is still being put out."""
    from baranet_bdml_b200 import _lib
    rng = np.random.default_rng(B + S)
    n, eps, scale = S + n_old, 1e-5, 4.0 * E ** -0.5
    q, k = rng.standard_normal((B, S, H, E)), R.unit_rms(rng.standard_normal((B, n, G, E)), eps)
    qg, kg, vg = _pad(q, dtype), _pad(k, dtype), _pad(rng.standard_normal((B, n, G, V)), dtype)
    V8, E8 = vg.shape[-1] // G, kg.shape[-1] // G
    seqs = [0, B // 2, B - 1]
    heads = [0, H // 2, H - 1]
    for bound in (0.0, 1.02 * E * scale):
        out = torch.full((B, S, H * V8), 7.0, dtype=dtype, device="cuda")
        word = torch.zeros(1, dtype=torch.int32, device="cuda")
        for _ in range(3):
            _lib.check(_lib.load().bn_attn_chunked(
                qg.data_ptr(), H * E8, kg.data_ptr(), G * E8, vg.data_ptr(), G * V8, None, 0, out.data_ptr(), H * V8, B, S, n_old, n, H, G, E8,
                V8, chunk, E, eps, scale, bound, word.data_ptr(), code(dtype), stream()))
        torch.cuda.synchronize()
        assert int(word.item()) == 0
        Q, K_, V_, got = R.unit_rms(_unpad(qg, H, E), eps), _unpad(kg, G, E), _unpad(vg, G, V), _unpad(out, H, V)
        for b in seqs:
            for h in heads:
                g = h // (H // G)
                Qb = np.concatenate([np.zeros((n_old, 1, E)), Q[b, :, h:h + 1]])
                want = R.chunked_attention(Qb, K_[b, :, g:g + 1], V_[b, :, g:g + 1], scale, chunk)[n_old:, 0]
                assert np.abs(got[b, :, h] - want).max() <= (2e-5 if dtype == torch.float32 else 3e-2), (bound, b, h)


@DTYPES
@pytest.mark.parametrize("chunk,n_old", [(70, 0), (70, 69), (128, 5), (200, 131)])
def test_keys_just_inside_and_outside_a_chunk(lib, dtype, chunk, n_old):
    """One key that every query of its chunk picks out (its score is 8 standard deviations up): the first and the last of a
    chunk, and far ones.  Its value stands at the queries of its own chunk behind it and nowhere else."""
    rng = np.random.default_rng(chunk)
    H, G, E, V, n = 4, 2, 64, 64, 3 * chunk
    S = n - n_old
    u = R.unit_rms(rng.standard_normal(E), 0.0)
    for key in (0, chunk - 1, chunk, chunk + 1, 2 * chunk - 1, 2 * chunk, n - 2):
        k = R.unit_rms(rng.standard_normal((n, G, E)), 1e-5)
        k -= (k @ u)[..., None] * u / E
        k[key] = u
        v = rng.standard_normal((n, G, V)) * 0.1
        v[key] = 5.0
        q = np.tile(u * 0.3, (S, H, 1)) + 0.001 * rng.standard_normal((S, H, E))
        got, want = _chunked_attention(q, k, v, np.full((S, H, V), 20.0), n_old, chunk, 10.0 / E, 1e-5, dtype, bound=10.2)
        assert np.abs(got - want).max() <= (5e-5 if dtype == torch.float32 else 3e-2), key
        seen = np.array([i >= key and i // chunk == key // chunk for i in range(n_old, n)])
        if seen.any():
            assert got[seen].min() > 4.0
        assert np.abs(got[~seen]).max() < 1.0


@pytest.mark.parametrize("S", [64, 300])
def test_chunked_attention_growing_scores(lib, S):
    """Scores that rise along the keys by far more than the rescale threshold."""
    rng = np.random.default_rng(0)
    q = np.abs(rng.standard_normal((S, 2, 64)))
    k = np.abs(rng.standard_normal((S, 1, 64))) * np.linspace(0.1, 6.0, S)[:, None, None]
    v = rng.standard_normal((S, 1, 64))
    for chunk in (S, 70):
        got, want = _chunked_attention(q, k, v, rng.standard_normal((S, 2, 64)), 0, chunk, 0.3, 1e-5, torch.bfloat16)
        assert np.abs(got - want).max() <= 3e-2


@DTYPES
@pytest.mark.parametrize("mixed", [False, True])
def test_keys_and_values_of_a_portion(lib, dtype, mixed):
    """Unit-RMS keys, mixed values, both to the portion's rows and to the cache rows of the chunk that it ends in; the tokens
    before the portion come back out of the cache."""
    from baranet_bdml_b200 import _lib
    from baranet_bdml_b200.kv_cache import ChunkCache
    rng = np.random.default_rng(3)
    B, G, E, V, chunk, lam, eps = 2, 3, 10, 20, 12, 0.3, 1e-3
    L = _lib.load()
    for start, S in ((0, 5), (0, 30), (7, 5), (7, 6), (11, 1), (12, 24), (5, 2)):
        cache = ChunkCache(4, chunk, G, E, V, dtype)
        cache.k.fill_(9.0)
        cache.v.fill_(8.0)
        kin, vin, vf = (rng.standard_normal((B * S, G, d)) for d in (E, V, V))
        k, v, f = (_pad(a, dtype) for a in (kin, vin, vf))
        proj = torch.cat([k, v], dim=1).contiguous()
        n_old = start % chunk
        n = n_old + S
        ko = torch.zeros((B * n, k.shape[1]), dtype=dtype, device="cuda")
        vo = torch.zeros((B * n, v.shape[1]), dtype=dtype, device="cuda")
        seq, pos = ints([3, 1]), ints([start, start])
        if n_old:
            cache.gather(seq, pos, n_old, ko, vo, n)
        _lib.check(L.bn_kv_prep(proj.data_ptr(), proj.data_ptr() + k.shape[1] * proj.element_size(), proj.stride(0),
                                f.data_ptr() if mixed else None, f.stride(0), lam, seq.data_ptr(), pos.data_ptr(), B, S, G, cache.dim_ld,
                                cache.vdim_ld, E, eps, ko.data_ptr(), vo.data_ptr(), n, n_old, cache.k.data_ptr(), cache.v.data_ptr(), chunk,
                                chunk, code(dtype), stream()))
        torch.cuda.synchronize()
        kw = R.unit_rms(_unpad(k, G, E), eps).reshape(B, S, G, E)
        vw = _unpad(v, G, V)
        vw = (R.mix_values(vw, _unpad(f, G, V), lam) if mixed else vw).reshape(B, S, G, V)
        tol = 2e-6 if dtype == torch.float32 else 2.0 ** -7
        kg, vg = _unpad(ko, G, E).reshape(B, n, G, E), _unpad(vo, G, V).reshape(B, n, G, V)
        assert np.abs(kg[:, n_old:] - kw).max() <= tol * 4 and np.abs(vg[:, n_old:] - vw).max() <= tol * 4
        assert (kg[:, :n_old] == 9.0).all() and (vg[:, :n_old] == 8.0).all()
        ck, cv = f64(cache.k), f64(cache.v)
        last = (start + S - 1) // chunk
        for b, slot in enumerate((3, 1)):
            for r in range(chunk):
                p = last * chunk + r
                if start <= p < start + S:
                    assert np.abs(ck[slot, :, r, :E] - kw[b, p - start]).max() <= tol * 4
                    assert np.abs(cv[slot, :, r, :V] - vw[b, p - start]).max() <= tol * 4
                    assert (ck[slot, :, r, E:] == 0).all() and (cv[slot, :, r, V:] == 0).all()
                else:
                    assert (ck[slot, :, r] == 9.0).all() and (cv[slot, :, r] == 8.0).all()
        assert (ck[[0, 2]] == 9.0).all()


@DTYPES
@pytest.mark.parametrize("H,G,E,V,chunk", [(8, 2, 64, 64, 200), (4, 4, 48, 64, 130), (32, 2, 128, 128, 300), (5, 1, 10, 11, 7), (3, 1, 256, 256, 150),
                                           (40, 1, 24, 136, 64), (2, 1, 264, 40, 40), (6, 3, 72, 200, 1)])
def test_one_token_over_the_cache(lib, dtype, H, G, E, V, chunk):
    """One token per row against caches of one and of several chunks' age, rows in slots of their own, for every number of
    parts; the new key and value are appended, and nothing of what the rows held before is seen."""
    from baranet_bdml_b200 import _lib
    from baranet_bdml_b200.kv_cache import ChunkCache
    rng = np.random.default_rng(H + chunk)
    positions = [0, 1, chunk - 1, chunk, chunk + 1, 2 * chunk - 1, 3 * chunk + chunk // 2, 31, 32, 33, 63, 64]
    B, eps, lam, scale = len(positions), 1e-4, 0.4, 4.0 * E ** -0.5
    groups = -(-(H // G) // 16)
    L = _lib.load()
    best = L.bn_gqa_step_splits(B, H, G, -(-E // 8) * 8, -(-V // 8) * 8, chunk, code(dtype))
    for mixed, splits in ((True, 1), (False, 2), (True, 3), (True, best), (False, 64)):
        cache = ChunkCache(B + 2, chunk, G, E, V, dtype, groups=groups)
        cache.k.fill_(9.0)                                  # stale rows must not be seen
        cache.v.fill_(9.0)
        slots = rng.permutation(B + 2)[:B]
        keys, vals = [], []
        for s, p in zip(slots, positions):
            m = p % chunk
            kk, vv = R.unit_rms(rng.standard_normal((m + 1, G, E)), eps), rng.standard_normal((m + 1, G, V))
            cache.k[int(s), :, :m], cache.v[int(s), :, :m] = 0, 0
            cache.k[int(s), :, :m, :E] = gpu(kk[:m].transpose(1, 0, 2), dtype)
            cache.v[int(s), :, :m, :V] = gpu(vv[:m].transpose(1, 0, 2), dtype)
            keys.append(kk)
            vals.append(vv)
        q, g = rng.standard_normal((B, H, E)) * 2, 2 * rng.standard_normal((B, H, V))
        knew, vnew, vf = 3 * rng.standard_normal((B, G, E)), rng.standard_normal((B, G, V)), rng.standard_normal((B, G, V))
        parts = [_pad(a, dtype) for a in (q, knew, vnew, g)]
        proj, f = torch.cat(parts, dim=1).contiguous(), _pad(vf, dtype)
        at = np.cumsum([0] + [t.shape[1] for t in parts]) * proj.element_size()
        out = torch.full((B, H * cache.vdim_ld), 7.0, dtype=dtype, device="cuda")
        partial = torch.full((B * G * groups * splits * 16 * (cache.vdim_ld + 2),), 5.0, device="cuda")
        sl, ps, word = ints(slots), ints(positions), torch.zeros(1, dtype=torch.int32, device="cuda")
        _lib.check(L.bn_gqa_step(
            *(int(proj.data_ptr() + a) for a in at[:4]), proj.stride(0), f.data_ptr() if mixed else None, f.stride(0), lam, cache.k.data_ptr(),
            cache.v.data_ptr(), cache.num_seqs, cache.ring_tokens, chunk, sl.data_ptr(), ps.data_ptr(), partial.data_ptr(),
            cache.tickets.data_ptr(), splits, out.data_ptr(), out.stride(0), B, H, G, cache.dim_ld, cache.vdim_ld, E, eps, scale,
            word.data_ptr(), code(dtype), stream()))
        torch.cuda.synchronize()
        assert int(word.item()) == 0 and int(cache.tickets.abs().sum()) == 0
        got = _unpad(out, H, V)
        kn, vn = R.unit_rms(_unpad(parts[1], G, E), eps), _unpad(parts[2], G, V)
        if mixed:
            vn = R.mix_values(vn, _unpad(f, G, V), lam)
        Q, gate = R.unit_rms(_unpad(parts[0], H, E), eps), R.sigmoid(_unpad(parts[3], H, V))
        for b, (s, p) in enumerate(zip(slots, positions)):
            m = p % chunk
            kk = np.concatenate([f64(gpu(keys[b][:m], dtype)), kn[b:b + 1]])
            vv = np.concatenate([f64(gpu(vals[b][:m], dtype)), vn[b:b + 1]])
            Qb = np.concatenate([np.zeros((m, H, E)), Q[b:b + 1]])
            want = R.chunked_attention(Qb, kk, vv, scale, m + 1)[m] * gate[b]
            assert np.abs(got[b] - want).max() <= (3e-5 if dtype == torch.float32 else 3e-2), (b, p, splits)
            tol = 1e-5 if dtype == torch.float32 else 2.0 ** -6
            assert np.abs(f64(cache.k[int(s), :, m, :E]) - kn[b]).max() <= tol and np.abs(f64(cache.v[int(s), :, m, :V]) - vn[b]).max() <= tol
            assert (f64(cache.k[int(s), :, m + 1:]) == 9.0).all()


@DTYPES
def test_a_token_behind_the_cache_gives_nan_and_touches_nothing(lib, dtype):
    from baranet_bdml_b200.mixers import ChunkedAttention, ChunkedAttentionConfig
    w = K.weights(K.config([K.layer(K.attention(dim=16, vdim=16, chunk=50))], 56, 16, 1), 1)
    mixer = ChunkedAttention(ChunkedAttentionConfig(6, 2, 16, 16, 50, 0.5, True), 56, 1e-5, lambda n, *s: w["l0.mix." + n], dtype)
    cache = mixer.new_state(2, 20)
    proj = mixer.project(torch.ones((2, 56), dtype=dtype, device="cuda"))
    out = mixer(proj, 2, 1, cache, ints([0, 1]), ints([20, 19]), None)
    assert bool(out[0].isnan().all()) and not bool(out[1].isnan().any())
    assert float(cache.k[0].float().abs().sum()) == 0 and float(cache.k[1, :, 19].float().abs().sum()) > 0


@DTYPES
@pytest.mark.parametrize("sizes", [dict(), dict(heads=2, kv_heads=2, dim=64, vdim=128, chunk=64), dict(heads=4, kv_heads=1, dim=5, vdim=3, chunk=2),
                                   dict(heads=17, kv_heads=1, dim=16, vdim=8, chunk=141), dict(heads=2, kv_heads=1, dim=320, vdim=264, chunk=33)])
def test_attention_mixer_alone(lib, dtype, sizes):
    """A mixer over rows of its own choosing, cut in several ways, two sequences with different inputs and first values."""
    from baranet_bdml_b200.mixers import ChunkedAttention, ChunkedAttentionConfig
    m = K.attention(**sizes)
    w = K.weights(K.config([K.layer(m)], 56, 16, 1), 11)
    W = K.as_f64(w)
    cfg = ChunkedAttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"], m["scale"], True)
    mixer = ChunkedAttention(cfg, 56, 1e-5, lambda name, *shape: w["l0.mix." + name], dtype)
    T, B = 140, 2
    rng = np.random.default_rng(12)
    h = gpu(rng.standard_normal((B, T, 56)), dtype)
    vf = rng.standard_normal((B, T, m["kv_heads"], m["vdim"]))
    f = _pad(vf, dtype)
    for mixed in (True, False):
        want = np.stack([R.attention(f64(h[b]), lambda s: W["l0.mix." + s], m, 1e-5,
                                     _unpad(f[b], m["kv_heads"], m["vdim"]) if mixed else None)[0] for b in range(B)])
        for cut in ([T], [3, 1, 64, 2, 1, 69], [70] + [1] * 70, [1, 2] * 46 + [2]):
            st = mixer.new_state(2)
            got, at = [], 0
            for n in cut:
                pos = ints([at] * B)
                proj = mixer.project(h[:, at:at + n].reshape(B * n, 56).contiguous())
                first = f[:, at:at + n].reshape(B * n, -1).contiguous() if mixed else None
                y = mixer(proj, B, n, st, ints([1, 0]), pos, None if n == 1 else at, first)
                got.append(f64(y)[:, :56].reshape(B, n, 56))
                at += n
            assert at == T
            assert K.error(np.concatenate(got, axis=1), want) <= (2e-5 if dtype == torch.float32 else 3e-2), cut[:6]
