"""Soluzen without a GPU: reading configurations and checkpoints, the order of layer runs, slots, and that the plain
restatement of its mechanisms agrees with other ways of writing them."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import soluzen_cases as K
from oracle import ref_soluzen as R

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", list(K.CASES))
def test_config_and_layer_runs(name):
    from baranet_bdml_b200.soluzen import SoluzenConfig
    raw = K.CASES[name]
    c = SoluzenConfig.from_dict(json.loads(json.dumps(raw)))
    assert c.runs() == R.schedule(raw)
    assert (c.width, c.vocab_size, c.side_dim, c.eps) == (raw["width"], raw["vocab"], raw["token_side"]["dim"], raw["norm"]["eps"])
    for lc, lay in zip(c.layers, raw["layers"]):
        assert lc.kind == lay["type"] and lc.ff == (None if lay["mlp"] is None else lay["mlp"]["ff"])
        if lc.kind == "latent_attention":
            assert lc.mixer.window == lay["mixer"]["mask"]["size"] and lc.mixer.scale == lay["mixer"]["scale"]
            assert lc.mixer.rope_base == lay["mixer"]["rot"]["base"]
        else:
            assert lc.mixer.taps == lay["mixer"]["conv"] and lc.mixer.groups == lay["mixer"]["groups"]


def test_loop_order():
    c = K.config([K.layer(K.mamba())] * 4, 8, 8, 8, loop=(1, 3, 2))
    assert R.schedule(c) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0].update(mlp={"kind": "experts", "ff": 8}),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4),
    lambda c: c["loop"].update(stop=9),
    lambda c: c["layers"][0]["mixer"].update(groups=4)])
def test_config_refuses_what_it_does_not_know(change):
    from baranet_bdml_b200.soluzen import SoluzenConfig
    c = json.loads(json.dumps(K.CASES["odd"]))
    change(c)
    with pytest.raises(ValueError):
        SoluzenConfig.from_dict(c)


def test_safetensors_round_trip(tmp_path):
    from baranet_bdml_b200.checkpoint import Weights, read_safetensors, write_safetensors
    rng = np.random.default_rng(0)
    t = {"a": torch.from_numpy(rng.standard_normal((3, 5)).astype(np.float32)).to(torch.bfloat16),
         "b.c": torch.from_numpy(rng.integers(-9, 9, (7,)).astype(np.int32)), "d": torch.randn(2, 1, 3)}
    write_safetensors(str(tmp_path / "m.safetensors"), t)
    r = read_safetensors(str(tmp_path / "m.safetensors"))
    assert set(r) == set(t) and all(r[k].dtype == t[k].dtype and torch.equal(r[k], t[k]) for k in t)
    w = Weights(r)
    w("a", 3, 5)
    assert w.leftover() == ["b.c", "d"]
    with pytest.raises(RuntimeError, match="no tensor"):
        w("missing")
    with pytest.raises(RuntimeError, match="shape"):
        w("d", 2, 3)


def test_registry_names_and_dtypes():
    from baranet_bdml_b200 import build, registry
    assert set(registry.ARCHITECTURES) == {"LLaMA", "Soluzen", "Duponex"}
    with pytest.raises(RuntimeError, match="unknown architecture"):
        registry.build_model({"architecture": "nothing"}, None)
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model("/nonexistent", "float16")
    for sources in build.FAMILIES.values():
        assert set(sources) <= set(build.SOURCES)


def test_a_family_library_stands_alone(tmp_path, lib):
    """The library a single model family is served from links and exports what that family calls."""
    import ctypes
    from baranet_bdml_b200 import build
    path = build._build(build.FAMILIES["soluzen"], str(tmp_path / "family.so"), False, False, [])
    so = ctypes.CDLL(path)
    for name in ("bn_latent_prep", "bn_attn_window", "bn_latent_decode", "bn_ssm_scan", "bn_mamba2_step", "bn_residual_norm",
                 "bn_gemm_glu_bf16_nt", "bn_mm_f32", "bn_argmax_rows_f32"):
        assert hasattr(so, name), name


def test_bad_arguments_come_back_as_status(lib):
    from baranet_bdml_b200 import _lib
    assert lib.bn_residual_norm(None, None, 0, 0, None, 0.0, None, None, None, 0, 0, None, None, None, 0, 0, 0, 1, 8, 1e-5, None) == \
        _lib.BN_ERR_INVALID_ARG
    assert lib.bn_latent_decode_splits(0, 4, 64, 32, 128, 1) == 0
    assert lib.bn_latent_decode_splits(1, 4, 64, 32, 128, 0) >= 1
    assert lib.bn_ssm_scan(None, 0, None, None, None, None, None, 1, 1, 1, 1, 1, 1, None, 0, 0, None) == _lib.BN_ERR_INVALID_ARG


def test_slots_are_reset_and_run_out():
    from baranet_bdml_b200.kv_cache import RecurrentState, SequenceSlots
    st = RecurrentState(2, 1, 2, 3, 4, 2, device="cpu")
    slots = SequenceSlots(2, [st], device="cpu")
    a, b = slots.acquire(), slots.acquire()
    assert sorted((a, b)) == [0, 1]
    with pytest.raises(RuntimeError, match="in use"):
        slots.acquire()
    st.state.fill_(3.0)
    st.conv.fill_(2.0)
    slots.lens.fill_(9)
    slots.release(a)
    with pytest.raises(RuntimeError, match="not in use"):
        slots.release(a)
    assert slots.acquire() == a
    assert float(st.state[a].abs().sum()) == 0 and float(st.conv[a].abs().sum()) == 0 and int(slots.lens[a]) == 0
    assert float(st.state[b].min()) == 3.0 and int(slots.lens[b]) == 9


def test_command_line_help_and_errors():
    run = lambda *a: subprocess.run([sys.executable, "-m", "baranet_bdml_b200", *a], cwd=ROOT, capture_output=True, text=True, timeout=120)  # noqa: E731
    assert run().returncode == 2 and "generate" in run().stderr
    assert run("generate", "--help").returncode == 0
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--help"], capture_output=True, text=True, timeout=120)
    assert r.returncode == 0 and "--max-tokens" in r.stdout


# ------------------------------------------------------------------ the restatement itself
def test_recurrence_equals_its_quadratic_form():
    """The scan against y_i = sum_j exp(sum of decays j+1..i) dt_j (C_i . B_j) x_j + D x_i."""
    rng = np.random.default_rng(1)
    T, H, P, G, N = 9, 4, 3, 2, 5
    x, B, C = rng.standard_normal((T, H, P)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, A, D = rng.random((T, H)), -rng.random(H), rng.standard_normal(H)
    want = np.zeros((T, H, P))
    for h in range(H):
        for i in range(T):
            for j in range(i + 1):
                want[i, h] += np.exp(A[h] * dt[j + 1:i + 1, h].sum()) * dt[j, h] * (C[i, h // 2] @ B[j, h // 2]) * x[j, h]
            want[i, h] += D[h] * x[i, h]
    assert np.abs(R.selective_scan(x, B, C, dt, A, D) - want).max() < 1e-12


def test_rotation_depends_on_distance_only_and_window_counts_itself():
    rng = np.random.default_rng(2)
    q, k = rng.standard_normal((1, 8)), rng.standard_normal((1, 8))
    dot = lambda a, b: float((R.rotate_interleaved(q, [a], 100.0) * R.rotate_interleaved(k, [b], 100.0)).sum())   # noqa: E731
    assert abs(dot(7, 3) - dot(1007, 1003)) < 1e-9
    v = np.eye(5)[:, None, :]
    o = R.windowed_softmax_attention(np.zeros((5, 1, 2)), np.zeros((5, 1, 2)), v, 1.0, 3)[:, 0]
    assert np.allclose(o[4], [0, 0, 1 / 3, 1 / 3, 1 / 3]) and np.allclose(o[1], [0.5, 0.5, 0, 0, 0])


def test_convolution_taps_and_groups_of_the_norm():
    x = np.arange(1.0, 5.0)[:, None]
    assert np.allclose(R.causal_conv(x, np.array([[100.0, 10.0, 1.0]]), np.array([0.5]))[:, 0], [1.5, 12.5, 123.5, 234.5])
    y = np.array([[3.0, 4.0, 30.0, 40.0]])
    z = np.full((1, 4), 50.0)
    assert np.allclose(R.gated_group_norm(y, z, np.ones(4), 2, 0.0), np.array([[3, 4, 3, 4]]) / np.sqrt(12.5))
