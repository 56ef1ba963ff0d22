"""Duponex without a GPU: reading configurations, how the streams' matrices are folded, the cache's bookkeeping, that the plain
restatement of its mechanisms agrees with other ways of writing them, and that mistakes planted in it move its logits by a
hundred times what the GPU tests allow in fp32."""
import ctypes
import json

import numpy as np
import pytest
import torch

import duponex_cases as K
from oracle import ref_duponex as R


@pytest.mark.parametrize("name", list(K.CASES))
def test_config(name):
    from baranet_bdml_b200.duponex import DuponexConfig
    raw = K.CASES[name]
    c = DuponexConfig.from_dict(json.loads(json.dumps(raw)))
    assert (c.width, c.vocab_size, c.eps, c.streams) == (raw["width"], raw["vocab"], raw["norm"]["eps"], raw["streams"])
    assert (c.embedding_scale, c.residual_mult) == (raw["embedding"]["scale"], raw["residual_mult"])
    for lc, lay in zip(c.layers, raw["layers"], strict=True):
        m = lay["mixer"]
        assert lc.ff == (None if lay["mlp"] is None else lay["mlp"]["ff"])
        assert (lc.mixer.heads, lc.mixer.kv_heads, lc.mixer.dim, lc.mixer.vdim) == (m["heads"], m["kv_heads"], m["dim"], m["vdim"])
        assert (lc.mixer.chunk, lc.mixer.scale, lc.mixer.mixes_values) == (m["mask"]["size"], m["scale"], m["v_mix"])


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="mamba2"),
    lambda c: c["layers"][0].update(mlp={"kind": "experts", "ff": 8}),
    lambda c: c["layers"][0]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][2]["mixer"].update(vdim=12),
    lambda c: c.update(streams=0)])
def test_config_refuses_what_it_does_not_know(change):
    from baranet_bdml_b200.duponex import DuponexConfig
    c = json.loads(json.dumps(K.CASES["odd"]))
    change(c)
    with pytest.raises(ValueError):
        DuponexConfig.from_dict(c)


def test_folded_streams_read_the_same_sum():
    from baranet_bdml_b200.ops import StreamMix
    rng = np.random.default_rng(0)
    mix, out, read = rng.standard_normal((3, 4)), rng.standard_normal(4), rng.standard_normal(4)
    x, y = rng.standard_normal((3, 5)), rng.standard_normal(5)
    want = read @ (mix.T @ x + out[:, None] * y)
    full, folded = StreamMix(mix.tolist(), out, read), StreamMix(mix.tolist(), out, read, keep=False)
    assert (full.n_in, full.n_out, folded.n_in, folded.n_out) == (3, 4, 3, 1)
    assert np.allclose(np.array(full.mix).reshape(3, 4), mix, atol=1e-6) and np.allclose(np.array(full.w_out), out, atol=1e-6)
    got = np.array(folded.mix).reshape(3, 1).T @ x + np.array(folded.w_out)[:, None] * y
    assert np.allclose(folded.w_in[0] * got[0], want, atol=1e-5)


def test_heads_are_padded_with_zeros():
    from baranet_bdml_b200.mixers import pad_heads
    w = torch.arange(1.0, 31.0).reshape(6, 5)                       # two heads of three rows
    p = pad_heads(w, 2, 3)
    assert p.shape == (16, 5) and torch.equal(p[0:3], w[:3]) and torch.equal(p[8:11], w[3:])
    assert float(p[3:8].abs().sum() + p[11:].abs().sum()) == 0
    assert torch.equal(pad_heads(torch.arange(16.0), 2, 8), torch.arange(16.0))


def test_cache_sizes_and_slots():
    from baranet_bdml_b200.kv_cache import ChunkCache, SequenceSlots
    assert ChunkCache(2, 100, 3, 10, 20, device="cpu").k.shape == (2, 3, 100, 16)
    c = ChunkCache(2, 100, 3, 10, 20, max_tokens=40, device="cpu")
    assert c.ring_tokens == 40 and c.v.shape == (2, 3, 40, 24)
    assert ChunkCache(2, 8, 3, 10, 20, max_tokens=40, device="cpu").ring_tokens == 8
    slots = SequenceSlots(2, [c], device="cpu")
    a = slots.acquire()
    slots.lens[a] = 5
    slots.release(a)
    assert slots.acquire() == a and int(slots.lens[a]) == 0
    assert len(slots.tensors()) == 3


def test_a_family_library_stands_alone(tmp_path, lib):
    """The library a Duponex model is served from in a checkout without built files links and exports what it calls."""
    from baranet_bdml_b200 import build
    so = ctypes.CDLL(build._build(build.FAMILIES["duponex"], str(tmp_path / "family.so"), False, False, []))
    for name in ("bn_hyper_norm", "bn_kv_prep", "bn_kv_gather", "bn_attn_chunked", "bn_gqa_step", "bn_gqa_step_splits", "bn_bias_act_f32",
                 "bn_gemm_bias_act_bf16_nt", "bn_gemm_bias_act_bf16_nt_small_m", "bn_gemm_bias_act_bf16_nt_skinny", "bn_mm_f32",
                 "bn_embedding_gather_bf16", "bn_gemm_bf16_nt_f32", "bn_argmax_rows_f32"):
        assert hasattr(so, name), name


def test_bad_arguments_come_back_as_status(lib):
    from baranet_bdml_b200 import _lib
    assert lib.bn_hyper_norm(None, 1, 1, None, None, None, None, 0, None, None, None, None, 0, 0, 1, 8, 1e-5, None) == _lib.BN_ERR_INVALID_ARG
    assert lib.bn_gqa_step_splits(1, 6, 4, 16, 16, 10, 1) == 0                 # 6 heads over 4
    assert lib.bn_gqa_step_splits(1, 6, 2, 12, 16, 10, 1) == 0                 # not a multiple of 8
    assert lib.bn_gqa_step_splits(1, 6, 2, 16, 16, 10, 0) == 1
    assert 1 < lib.bn_gqa_step_splits(1, 8, 2, 64, 64, 100000, 1) <= 64
    buf = (ctypes.c_float * 64)()
    p = ctypes.addressof(buf) // 16 * 16 + 16
    # a portion whose old tokens reach behind the chunk's start; more tokens than rows
    for n_old, rows in ((7, 20), (0, 3)):
        assert lib.bn_attn_chunked(p, 8, p, 8, p, 8, None, 0, p, 8, 1, 4, n_old, rows, 1, 1, 8, 8, 7, 0, 0.0, 1.0, 0.0, None, 0, None) == \
            _lib.BN_ERR_INVALID_ARG


# ------------------------------------------------------------------ the restatement itself
def test_chunks_are_counted_from_position_zero():
    v = np.eye(7)[:, None, :]
    o = R.chunked_attention(np.zeros((7, 1, 2)), np.zeros((7, 1, 2)), v, 1.0, 3)[:, 0]
    for i in range(7):
        want = np.zeros(7)
        want[i // 3 * 3:i + 1] = 1 / (i - i // 3 * 3 + 1)
        assert np.allclose(o[i], want)


def test_query_heads_share_key_heads_in_blocks():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((5, 6, 4)), rng.standard_normal((5, 2, 4)), rng.standard_normal((5, 2, 3))
    o = R.chunked_attention(q, k, v, 0.7, 5)
    for h, g in enumerate([0, 0, 0, 1, 1, 1]):
        assert np.allclose(o[:, h:h + 1], R.chunked_attention(q[:, h:h + 1], k[:, g:g + 1], v[:, g:g + 1], 0.7, 5))


def test_streams_are_indexed_from_to():
    s = np.array([[[1.0]], [[10.0]]])
    new = R.write_streams(s, np.array([[1.0, 2.0], [3.0, 4.0]]), np.array([100.0, 200.0]), np.array([[1.0]]))
    assert new[:, 0, 0].tolist() == [1 + 30 + 100, 2 + 40 + 200]
    assert R.read_streams(s, np.array([2.0, 0.5]))[0, 0] == 7.0
    assert np.allclose(R.squared_relu(np.array([-2.0, 0.0, 3.0])), [0, 0, 9]) and np.isclose(R.sigmoid(np.log(3.0)), 0.75)
    assert np.allclose(R.unit_rms(np.array([3.0, 4.0]), 0.0), np.array([3.0, 4.0]) / np.sqrt(12.5))


def test_planted_mistakes_are_far_beyond_the_fp32_gate():
    cfg = K.CASES["odd"]
    W, toks = K.as_f64(K.weights(cfg, 0)), np.random.default_rng(5).integers(0, cfg["vocab"], 61)
    want = R.forward(cfg, W, toks)

    def mistaken(change):
        c, V = json.loads(json.dumps(cfg)), dict(W)
        change(c, V)
        return np.quantile(K.row_errors(R.forward(c, V, toks), want), 0.8)
    size = lambda i, n: (lambda c, V: c["layers"][i]["mixer"]["mask"].update(size=n))      # noqa: E731
    scaled = lambda name, f: (lambda c, V: V.update({name: V[name] * f}))                  # noqa: E731
    for change in (size(0, 8), size(0, 6), size(1, 18), size(1, 20), size(2, 15), size(2, 17), scaled("l1.ls1", 0), scaled("l2.ls2", 1.5),
                   scaled("l0.mix.q.b", 0), scaled("l0.mix.k.b", 0), scaled("l2.mix.v.b", 0), scaled("l0.mix.o.b", 0), scaled("l3.mix.g", 0),
                   scaled("l2.mix.vmix", 0), scaled("l3.mix.vmix", 0), lambda c, V: V.update({"l1.hc1.mix": V["l1.hc1.mix"].T}),
                   lambda c, V: V.update({"l2.hc2.in": V["l2.hc2.in"][::-1]}), lambda c, V: V.update({"l0.hc2.out": V["l0.hc2.out"] * [0.3, 1.0, 1.0]}),
                   lambda c, V: c.update(residual_mult=0.4), lambda c, V: c["embedding"].update(scale=1.4),
                   lambda c, V: c["layers"][2]["mixer"].update(v_mix=False)):
        assert mistaken(change) > 1e-2
