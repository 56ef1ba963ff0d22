"""Sublayers of the models that are served from per-sequence slots, in fp32 and in bf16: latent attention with a sliding
window, grouped-query attention in chunks, the Mamba-2 mixer, MLPs with a choice of activation, and the per-layer token
input.  Sizes and constants are parameters; weights come from a function name -> tensor.

A mixer is called with the rows of B sequences x S new tokens: `seq_ids` (B) are the sequences' slots in its cache or state
(which `new_state` makes), `positions` (B) the position of each one's first new token, both int32 on the GPU.  `n_old` is how
many earlier tokens every one of the B sequences has; None with S = 1 selects the one-token kernels, for which the sequences'
lengths may differ.  Inference only."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Optional

import torch

from . import _lib, ops
from .kv_cache import ChunkCache, LatentRingCache, RecurrentState
from .ops import _dt, _ptr, _stream, round8


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int                # unrotated query / key columns per head
    rot_dim: int            # rotated ones
    vdim: int
    q_rank: int
    kv_rank: int
    window: int             # a position sees itself and the window - 1 before it
    rope_base: float
    scale: float

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim, self.q_rank, self.kv_rank, self.window) <= 0 or self.rot_dim < 0 or self.rot_dim % 2:
            raise ValueError(f"latent attention: bad sizes {self}")


class LatentAttention:
    """Queries through a normalised latent of q_rank; keys and values expanded from a normalised latent of kv_rank that is
    all the cache holds, beside one rotated key part shared by the heads."""

    def __init__(self, cfg: LatentAttentionConfig, width: int, eps: float, weight: Callable, dtype):
        c, H = cfg, cfg.heads
        self.cfg, self.dtype, self.eps = cfg, dtype, float(eps)
        dkv = weight("dkv", c.kv_rank + c.rot_dim, width)
        self.down = ops.Linear(torch.cat([weight("dq", c.q_rank, width), dkv]), dtype)      # [c_q | c | rotated key part]
        self.q_norm = ops.NormWeight(weight("dq.norm", c.q_rank), None, eps)
        self.kv_norm = ops.NormWeight(weight("dkv.norm", c.kv_rank), None, eps)
        self.uq = ops.Linear(weight("uq", H * (c.dim + c.rot_dim), c.q_rank), dtype)
        self.ukv = ops.Linear(torch.cat([weight("uk", H * c.dim, c.kv_rank), weight("uv", H * c.vdim, c.kv_rank)]), dtype)
        self.uk, self.uv = self.ukv.weight[:H * c.dim], self.ukv.weight[H * c.dim:]
        self.o = ops.Linear(weight("o", width, H * c.vdim), dtype)
        self.freq = ops.rotation_frequencies(c.rot_dim, c.rope_base)
        self.kv_ld, self.rot_ld = round8(c.kv_rank), round8(c.rot_dim)

    def new_state(self, num_seqs: int) -> LatentRingCache:
        c = self.cfg
        return LatentRingCache(num_seqs, c.window, c.kv_rank, c.rot_dim, self.dtype)

    def _prep(self, proj, B, S, cache, seq_ids, positions, latents, keys, rows_per_seq, row_offset):
        c = self.cfg
        cq = torch.empty((B * S, self.uq.k), dtype=self.dtype, device=proj.device)
        _lib.check(_lib.load().bn_latent_prep(
            proj.data_ptr(), proj.stride(0), self.q_norm.weight.data_ptr(), self.kv_norm.weight.data_ptr(), self.eps,
            self.freq.data_ptr(), seq_ids.data_ptr(), positions.data_ptr(), B, S, c.q_rank, c.kv_rank, c.rot_dim, cq.data_ptr(),
            self.uq.k, _ptr(latents), _ptr(keys), rows_per_seq, row_offset, cache.ring.data_ptr(), cache.ring_tokens,
            _dt(self.dtype), _stream()))
        return cq

    def __call__(self, h: torch.Tensor, B: int, S: int, cache: LatentRingCache, seq_ids, positions, n_old: Optional[int]):
        proj = self.down(h)
        out = torch.empty((B * S, self.o.k), dtype=self.dtype, device=h.device)
        if n_old is None:
            self._one_token(proj, B, cache, seq_ids, positions, out)
        else:
            self._portion(proj, B, S, cache, seq_ids, positions, n_old, out)
        return self.o(out)

    def _portion(self, proj, B, S, cache, seq_ids, positions, n_old, out):
        c, dev = self.cfg, proj.device
        n_old = min(n_old, c.window - 1)                      # what the portion's first token still sees
        n = n_old + S
        latents = torch.empty((B * n, self.kv_ld), dtype=self.dtype, device=dev)
        keys = torch.empty((B * n, self.rot_ld), dtype=self.dtype, device=dev)
        if n_old:                                             # before the portion's own rows replace any in the ring
            cache.gather(seq_ids, positions, n_old, latents, keys, n)
        cq = self._prep(proj, B, S, cache, seq_ids, positions, latents, keys, n, n_old)
        q = self.uq(cq)
        lib = _lib.load()
        _lib.check(lib.bn_rope_heads(q.data_ptr(), q.stride(0), B, S, c.heads, c.dim, c.rot_dim, self.freq.data_ptr(),
                                     positions.data_ptr(), _dt(self.dtype), _stream()))
        kv = self.ukv(latents)
        v_ptr = kv.data_ptr() + c.heads * c.dim * kv.element_size()
        _lib.check(lib.bn_attn_window(
            q.data_ptr(), q.stride(0), kv.data_ptr(), v_ptr, kv.stride(0), keys.data_ptr(), self.rot_ld, out.data_ptr(),
            out.stride(0), B, S, n_old, n, c.heads, c.dim, c.rot_dim, c.vdim, c.window, float(c.scale),
            ops.status_word(dev).data_ptr(), _dt(self.dtype), _stream()))

    def _one_token(self, proj, B, cache, seq_ids, positions, out):
        c, dev, dt = self.cfg, proj.device, _dt(self.dtype)
        lib, s = _lib.load(), _stream()
        cq = self._prep(proj, B, 1, cache, seq_ids, positions, None, None, 0, 0)
        q = self.uq(cq)
        q_abs = torch.empty((B, c.heads, self.kv_ld + self.rot_ld), dtype=self.dtype, device=dev)
        _lib.check(lib.bn_latent_absorb_q(q.data_ptr(), q.stride(0), self.uk.data_ptr(), self.freq.data_ptr(),
                                          positions.data_ptr(), q_abs.data_ptr(), B, c.heads, c.dim, c.rot_dim, c.kv_rank, dt, s))
        splits = lib.bn_latent_decode_splits(B, c.heads, c.kv_rank, c.rot_dim, c.window, dt)
        partial = torch.empty((B, c.heads, splits, self.kv_ld), dtype=torch.float32, device=dev)
        lse = torch.empty((B, c.heads, splits), dtype=torch.float32, device=dev)
        _lib.check(lib.bn_latent_decode(q_abs.data_ptr(), cache.ring.data_ptr(), cache.num_seqs, cache.ring_tokens, seq_ids.data_ptr(),
                                        positions.data_ptr(), partial.data_ptr(), lse.data_ptr(), splits, B, c.heads, c.kv_rank,
                                        c.rot_dim, c.window, float(c.scale), dt, s))
        _lib.check(lib.bn_latent_expand_out(partial.data_ptr(), lse.data_ptr(), splits, self.uv.data_ptr(), out.data_ptr(),
                                            out.stride(0), B, c.heads, c.vdim, c.kv_rank, dt, s))


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int                # per-head query / key columns
    vdim: int
    chunk: int              # a position sees its own chunk up to itself; chunks start at the multiples of this
    scale: float
    mixes_values: bool      # whether the layer takes part in value mixing

    def __post_init__(self):
        if min(self.heads, self.kv_heads, self.dim, self.vdim, self.chunk) <= 0 or self.heads % self.kv_heads:
            raise ValueError(f"chunked attention: bad sizes {self}")


def pad_heads(rows: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
    """(heads * dim, ...) -> (heads * round8(dim), ...), zeros behind each head: every head starts on a 16-byte boundary."""
    out = torch.zeros((heads, round8(dim)) + tuple(rows.shape[1:]), dtype=rows.dtype, device=rows.device)
    out[:, :dim] = rows.reshape((heads, dim) + tuple(rows.shape[1:]))
    return out.reshape((heads * round8(dim),) + tuple(rows.shape[1:]))


class ChunkedAttention:
    """Grouped-query attention in chunks of positions, unit-RMS queries and keys, no rotation, a sigmoid gate on the heads'
    outputs, biases on the projections, and values mixed with those of an earlier layer.

    `project` gives the rows [q | k | v | gate] that everything else reads; `values` is the v of them, which a later layer may
    take as `v_first`."""

    def __init__(self, cfg: ChunkedAttentionConfig, width: int, eps: float, weight: Callable, dtype):
        c = cfg
        self.cfg, self.dtype, self.eps = cfg, dtype, float(eps)
        self.dim_ld, self.vdim_ld = round8(c.dim), round8(c.vdim)
        self.head_groups = -(-(c.heads // c.kv_heads) // 16)                          # of 16 query heads per key head
        sizes = [("q", c.heads, c.dim), ("k", c.kv_heads, c.dim), ("v", c.kv_heads, c.vdim), ("g", c.heads, c.vdim)]
        w = [pad_heads(weight(n, h * d, width), h, d) for n, h, d in sizes]
        b = [pad_heads(weight(n + ".b", h * d), h, d) for n, h, d in sizes[:3]]
        b.append(torch.zeros(w[3].shape[0], dtype=b[0].dtype, device=b[0].device))                      # the gate has no bias
        self.proj = ops.Linear(torch.cat(w), dtype, bias=torch.cat(b))
        self.cols = [0]
        for part in w:
            self.cols.append(self.cols[-1] + part.shape[0])
        o = weight("o", width, c.heads * c.vdim)
        self.o = ops.Linear(pad_heads(o.t(), c.heads, c.vdim).t(), dtype, bias=weight("o.b", width))
        self.score_bound = 1.02 * c.dim * abs(c.scale)          # unit-RMS queries and keys, the keys rounded to bf16
        self.mix = float(weight("vmix").reshape(())) if c.mixes_values else 0.0      # one number

    def new_state(self, num_seqs: int, max_tokens: Optional[int] = None) -> ChunkCache:
        c = self.cfg
        return ChunkCache(num_seqs, c.chunk, c.kv_heads, c.dim, c.vdim, self.dtype, max_tokens, self.head_groups)

    def project(self, h: torch.Tensor) -> torch.Tensor:
        return self.proj(h)

    def values(self, proj: torch.Tensor) -> torch.Tensor:
        return proj[:, self.cols[2]:self.cols[3]]

    def __call__(self, proj: torch.Tensor, B: int, S: int, cache: ChunkCache, seq_ids, positions, n_old: Optional[int],
                 v_first: Optional[torch.Tensor] = None):
        c = self.cfg
        if v_first is not None and (v_first.dtype != self.dtype or tuple(v_first.shape) != (B * S, c.kv_heads * self.vdim_ld)):
            raise RuntimeError("chunked attention: the values to mix in must have this layer's heads and sizes")
        out = torch.empty((B * S, self.o.k), dtype=self.dtype, device=proj.device)
        (self._one_token if n_old is None else self._portion)(proj, B, S, cache, seq_ids, positions, n_old, v_first, out)
        return self.o(out)

    def _columns(self, proj):
        """pointers to the q, k, v and gate columns"""
        return [proj.data_ptr() + at * proj.element_size() for at in self.cols[:4]]

    def _portion(self, proj, B, S, cache, seq_ids, positions, n_old, v_first, out):
        c, dev, dt, lib, s = self.cfg, proj.device, _dt(self.dtype), _lib.load(), _stream()
        q, k, v, g = self._columns(proj)
        n_old %= c.chunk                                      # the tokens of the portion's first chunk that it still sees
        n = n_old + S
        keys = torch.empty((B * n, c.kv_heads * self.dim_ld), dtype=self.dtype, device=dev)
        values = torch.empty((B * n, c.kv_heads * self.vdim_ld), dtype=self.dtype, device=dev)
        if n_old:                                             # before the portion's own rows replace any in the cache
            cache.gather(seq_ids, positions, n_old, keys, values, n)
        _lib.check(lib.bn_kv_prep(
            k, v, proj.stride(0), _ptr(v_first), 0 if v_first is None else v_first.stride(0), self.mix, seq_ids.data_ptr(),
            positions.data_ptr(), B, S, c.kv_heads, self.dim_ld, self.vdim_ld, c.dim, self.eps, keys.data_ptr(), values.data_ptr(), n,
            n_old, cache.k.data_ptr(), cache.v.data_ptr(), cache.ring_tokens, c.chunk, dt, s))
        _lib.check(lib.bn_attn_chunked(
            q, proj.stride(0), keys.data_ptr(), keys.stride(0), values.data_ptr(), values.stride(0), g, proj.stride(0), out.data_ptr(),
            out.stride(0), B, S, n_old, n, c.heads, c.kv_heads, self.dim_ld, self.vdim_ld, c.chunk, c.dim, self.eps, float(c.scale),
            self.score_bound, ops.status_word(dev).data_ptr(), dt, s))

    def _one_token(self, proj, B, S, cache, seq_ids, positions, n_old, v_first, out):
        c, dev, dt, lib = self.cfg, proj.device, _dt(self.dtype), _lib.load()
        q, k, v, g = self._columns(proj)
        splits = lib.bn_gqa_step_splits(B, c.heads, c.kv_heads, self.dim_ld, self.vdim_ld, cache.ring_tokens, dt)
        partial = None
        if splits > 1:
            partial = torch.empty(B * c.kv_heads * self.head_groups * splits * 16 * (self.vdim_ld + 2), dtype=torch.float32, device=dev)
        _lib.check(lib.bn_gqa_step(
            q, k, v, g, proj.stride(0), _ptr(v_first), 0 if v_first is None else v_first.stride(0), self.mix, cache.k.data_ptr(),
            cache.v.data_ptr(), cache.num_seqs, cache.ring_tokens, c.chunk, seq_ids.data_ptr(), positions.data_ptr(), _ptr(partial),
            cache.tickets.data_ptr(), splits, out.data_ptr(), out.stride(0), B, c.heads, c.kv_heads, self.dim_ld, self.vdim_ld, c.dim,
            self.eps, float(c.scale), ops.status_word(dev).data_ptr(), dt, _stream()))


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int

    def __post_init__(self):
        if min(self.heads, self.vdim, self.state, self.groups, self.taps, self.norm_groups) <= 0 or self.heads % self.groups or \
                (self.heads * self.vdim) % self.norm_groups:
            raise ValueError(f"mamba2: bad sizes {self}")

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


class Mamba2Mixer:
    """Gated state-space mixer: projection, causal convolution, selective recurrence, gated group norm, projection."""

    def __init__(self, cfg: Mamba2Config, width: int, eps: float, weight: Callable, dtype):
        c = cfg
        self.cfg, self.dtype, self.eps = cfg, dtype, float(eps)
        f32 = lambda name, *shape: weight(name, *shape).to(device="cuda", dtype=torch.float32).contiguous()   # noqa: E731
        self.proj_in = ops.Linear(weight("in", c.inner + c.channels + c.heads, width), dtype)
        self.conv, self.conv_bias = f32("conv", c.channels, c.taps), f32("conv.b", c.channels)
        self.dt_bias, self.a_log, self.d = f32("dt_bias", c.heads), f32("A_log", c.heads), f32("D", c.heads)
        self.norm = f32("norm", c.inner)
        self.o = ops.Linear(weight("o", width, c.inner), dtype)

    def new_state(self, num_seqs: int) -> RecurrentState:
        c = self.cfg
        return RecurrentState(num_seqs, c.heads, c.vdim, c.state, c.channels, c.taps, self.dtype)

    def __call__(self, h: torch.Tensor, B: int, S: int, st: RecurrentState, seq_ids, positions, n_old: Optional[int]):
        c, dev, dt_code, lib, s = self.cfg, h.device, _dt(self.dtype), _lib.load(), _stream()
        rows = B * S
        proj = self.proj_in(h)
        out = torch.empty((rows, self.o.k), dtype=self.dtype, device=dev)
        if n_old is None:
            gated = torch.empty((rows, c.inner), dtype=torch.float32, device=dev)
            _lib.check(lib.bn_mamba2_step(
                proj.data_ptr(), proj.stride(0), self.conv.data_ptr(), self.conv_bias.data_ptr(), self.dt_bias.data_ptr(),
                self.a_log.data_ptr(), self.d.data_ptr(), st.conv.data_ptr(), st.state.data_ptr(), seq_ids.data_ptr(),
                positions.data_ptr(), B, c.heads, c.vdim, c.groups, c.state, c.taps, gated.data_ptr(), dt_code, s))
            y, y_dt, z, z_ld = gated, 0, None, 0
        else:
            xbc = torch.empty((rows, round8(c.channels)), dtype=self.dtype, device=dev)
            dt = torch.empty((rows, c.heads), dtype=torch.float32, device=dev)
            a = torch.empty((rows, c.heads), dtype=torch.float32, device=dev)
            _lib.check(lib.bn_mamba2_conv(
                proj.data_ptr(), proj.stride(0), self.conv.data_ptr(), self.conv_bias.data_ptr(), self.dt_bias.data_ptr(),
                self.a_log.data_ptr(), st.conv.data_ptr(), seq_ids.data_ptr(), positions.data_ptr(), B, S, c.heads, c.vdim,
                c.groups, c.state, c.taps, xbc.data_ptr(), xbc.stride(0), dt.data_ptr(), a.data_ptr(), dt_code, s))
            y = torch.empty((rows, round8(c.inner)), dtype=self.dtype, device=dev)
            _lib.check(lib.bn_ssm_scan(xbc.data_ptr(), xbc.stride(0), dt.data_ptr(), a.data_ptr(), self.d.data_ptr(),
                                       st.state.data_ptr(), seq_ids.data_ptr(), B, S, c.heads, c.vdim, c.groups, c.state,
                                       y.data_ptr(), y.stride(0), dt_code, s))
            y_dt, z, z_ld = dt_code, proj, proj.stride(0)
        _lib.check(lib.bn_gated_group_norm(y.data_ptr(), y.stride(0), y_dt, _ptr(z), z_ld, self.norm.data_ptr(), out.data_ptr(),
                                           out.stride(0), rows, c.inner, c.norm_groups, self.eps, dt_code, s))
        return self.o(out)


class GatedMLP:
    """down(act(gate x) * up x)"""

    def __init__(self, inter: int, width: int, act: str, weight: Callable, dtype):
        self.gate_up = ops.GatedLinear(weight("gate", inter, width), weight("up", inter, width), act, dtype)
        self.down = ops.Linear(weight("down", width, inter), dtype)

    def __call__(self, h: torch.Tensor) -> torch.Tensor:
        return self.down(self.gate_up(h))


class MLP:
    """down(act(up x))"""

    def __init__(self, inter: int, width: int, act: str, weight: Callable, dtype):
        self.up = ops.Linear(weight("up", inter, width), dtype, act=act)
        self.down = ops.Linear(weight("down", width, inter), dtype)

    def __call__(self, h: torch.Tensor) -> torch.Tensor:
        return self.down(self.up(h))


class TokenSide:
    """Per-layer token input: proj(act(gate x) * e), e the layer's part of a row that the token itself selects.  What the
    residual stream gets is its RMS norm, which the next residual_norm takes while it adds it."""

    def __init__(self, dim: int, width: int, eps: float, act: str, weight: Callable, dtype):
        self.act = act
        self.gate = ops.Linear(weight("gate", dim, width), dtype)
        self.proj = ops.Linear(weight("proj", width, dim), dtype)
        self.norm = ops.NormWeight(weight("norm", width), None, eps)

    def __call__(self, x: torch.Tensor, e: torch.Tensor) -> ops.Pending:
        return ops.Pending(self.proj(self.gate.act_mul(x, e, self.act)), self.norm)
