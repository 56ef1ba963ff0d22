"""Paged bf16 KV cache and single-token decode.

The reference has no cache: `generate()` recomputes the whole sequence for
every new token and keeps the last row (mygrad/llama/llama_model.py:136-144).
`PagedKVCache` supplies what that loop lacks — K (stored rotated) and V of the
earlier tokens — so that decoding one token reads each cached byte once.

Layout of the pool (one per layer):
    pool[page][kv_head][0 = K, 1 = V][16 tokens][head_dim]   bf16
`page_table[seq][logical_page]` names the pool page; pages of a sequence need
not be contiguous.
"""
from __future__ import annotations

from typing import Optional

import torch

from . import _lib
from .ops import Workspace, _need, _stream

PAGE_TOKENS = _lib.BN_PAGE_TOKENS


class PagedKVCache:
    def __init__(self, num_pages: int, num_seqs: int, max_pages_per_seq: int, num_kv_heads: int = 4,
                 head_dim: int = 64, theta: float = 10000.0, device="cuda"):
        self.num_pages, self.num_seqs, self.max_pages = int(num_pages), int(num_seqs), int(max_pages_per_seq)
        self.num_kv_heads, self.head_dim, self.theta = int(num_kv_heads), int(head_dim), float(theta)
        self.pool = torch.zeros((num_pages, num_kv_heads, 2, PAGE_TOKENS, head_dim), dtype=torch.bfloat16, device=device)
        self.page_table = torch.zeros((num_seqs, max_pages_per_seq), dtype=torch.int32, device=device)
        self.seq_lens = torch.zeros((num_seqs,), dtype=torch.int32, device=device)
        self._ws = {}          # decode scratch per (B, Hq, max_seq_len, chunk_tokens); kept while the cache lives

    @property
    def max_seq_len(self) -> int:
        return self.max_pages * PAGE_TOKENS

    def append(self, seq_ids: torch.Tensor, positions: torch.Tensor, k_new: torch.Tensor, v_new: torch.Tensor) -> None:
        """Writes tokens (sequence seq_ids[t], position positions[t]) with
        RoPE(K) fused; k_new, v_new (T, Hkv*D) fp32 or bf16.  Does not touch
        seq_lens (the caller advances them)."""
        T = k_new.shape[0]
        if k_new.dtype not in (torch.float32, torch.bfloat16) or v_new.dtype != k_new.dtype:
            raise RuntimeError("kv append: k/v must both be fp32 or both bf16")
        for t in (k_new, v_new):
            if not t.is_cuda:
                raise RuntimeError("kv append: only GPU implementation available")
            if t.stride(1) != 1 or t.stride(0) != k_new.stride(0):
                raise RuntimeError("kv append: k/v rows must be contiguous with equal row stride")
        _need(seq_ids, torch.int32, "kv append(seq_ids)")
        _need(positions, torch.int32, "kv append(positions)")
        _lib.check(_lib.load().bn_kv_append(
            self.pool.data_ptr(), self.num_pages, self.page_table.data_ptr(), self.max_pages, seq_ids.data_ptr(),
            positions.data_ptr(), T, k_new.data_ptr(), v_new.data_ptr(), k_new.stride(0),
            0 if k_new.dtype == torch.float32 else 1, self.num_kv_heads, self.head_dim, self.theta, _stream()))

    def workspace(self, B: int, Hq: int, max_seq_len: int, chunk_tokens: int = 0) -> Workspace:
        """The decode scratch for this shape.  A buffer, once handed out, is never freed or replaced while the
        cache lives: a captured CUDA graph may hold its address."""
        key = (B, Hq, max_seq_len, chunk_tokens)
        ws = self._ws.get(key)
        if ws is None:
            n = _lib.load().bn_attn_decode_workspace_bytes(B, Hq, self.num_kv_heads, self.head_dim, max_seq_len,
                                                          chunk_tokens)
            if n == 0:
                raise RuntimeError("bn_attn_decode_paged: unsupported shape")
            ws = self._ws[key] = Workspace(n, self.pool.device)
        return ws

    def status(self) -> None:
        """Raises if a decode launch on any of this cache's scratch buffers gave up on a bounded wait."""
        for ws in self._ws.values():
            ws.status()

    def decode(self, q: torch.Tensor, *, num_heads: int, scale: Optional[float] = None, rope_q: bool = True,
               q_positions: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
               out_f32: Optional[torch.Tensor] = None, lse: Optional[torch.Tensor] = None,
               max_seq_len: Optional[int] = None, chunk_tokens: int = 0, seq_lens: Optional[torch.Tensor] = None,
               page_table: Optional[torch.Tensor] = None) -> torch.Tensor:
        """q (B, Hq, D) bf16 (pre-RoPE when rope_q) -> out (B, Hq, D) bf16."""
        _need(q, torch.bfloat16, "decode(q)")
        B, Hq, D = q.shape
        seq_lens = self.seq_lens if seq_lens is None else seq_lens
        page_table = self.page_table if page_table is None else page_table
        if out is None and out_f32 is None:
            out = torch.empty_like(q)
        if max_seq_len is None:
            max_seq_len = self.max_seq_len
        if scale is None:
            scale = 1.0 / (D ** 0.5)
        ws = self.workspace(B, Hq, max_seq_len, chunk_tokens)
        _lib.check(_lib.load().bn_attn_decode_paged(
            q.data_ptr(), self.pool.data_ptr(), self.num_pages, page_table.data_ptr(), page_table.shape[1],
            seq_lens.data_ptr(), q_positions.data_ptr() if q_positions is not None else None,
            out.data_ptr() if out is not None else None, out_f32.data_ptr() if out_f32 is not None else None,
            lse.data_ptr() if lse is not None else None, B, Hq, self.num_kv_heads, D, float(scale), self.theta,
            int(bool(rope_q)), int(max_seq_len), int(chunk_tokens), ws.ptr, ws.nbytes, _stream()))
        return out if out is not None else out_f32


class LatentRingCache:
    """What latent attention keeps of a sequence's last tokens: the normalised latent and the rotated key part that all
    heads share.  A token's row is position % ring_tokens, so a sliding-window layer holds a constant amount per sequence
    however long the sequence gets: ring_tokens is the window, rounded up to whole pages of PAGE_TOKENS.

    ring[slot][ring_tokens][round8(kv_rank) | round8(rot_dim)], zeros behind the values of each part."""

    def __init__(self, num_seqs: int, window: int, kv_rank: int, rot_dim: int, dtype=torch.bfloat16, device="cuda"):
        from .ops import round8
        self.num_seqs, self.window, self.kv_rank, self.rot_dim, self.dtype = num_seqs, window, kv_rank, rot_dim, dtype
        self.kv_ld, self.rot_ld = round8(kv_rank), round8(rot_dim)
        self.ring_tokens = (window + PAGE_TOKENS - 1) // PAGE_TOKENS * PAGE_TOKENS
        self.ring = torch.zeros((num_seqs, self.ring_tokens, self.kv_ld + self.rot_ld), dtype=dtype, device=device)

    def reset(self, slot: int) -> None:
        """Nothing to clear: a row is read only for positions that the sequence itself has written."""

    def tensors(self):
        return [self.ring]

    def gather(self, seq_ids, positions, n_old: int, latents: torch.Tensor, keys: torch.Tensor, rows_per_seq: int) -> None:
        """The n_old tokens before `positions` to the first rows of each sequence's block of `latents` / `keys`."""
        from .ops import _dt
        _lib.check(_lib.load().bn_latent_gather(
            self.ring.data_ptr(), self.ring_tokens, self.kv_rank, self.rot_dim, seq_ids.data_ptr(), positions.data_ptr(),
            seq_ids.numel(), n_old, latents.data_ptr(), keys.data_ptr(), rows_per_seq, _dt(self.dtype), _stream()))


class ChunkCache:
    """Keys and values of a sequence's current chunk of positions, for attention that never looks behind a chunk's start: the
    token of position p in row p % chunk, so the next chunk overwrites the one before it.  `max_tokens` (the most tokens a
    sequence will have) bounds the rows where it is less than a chunk.

    k[slot][kv_head][ring_tokens][round8(dim)], v likewise, zeros behind the values."""

    def __init__(self, num_seqs: int, chunk: int, kv_heads: int, dim: int, vdim: int, dtype=torch.bfloat16,
                 max_tokens: Optional[int] = None, groups: int = 1, device="cuda"):
        from .ops import round8
        self.num_seqs, self.chunk, self.kv_heads, self.dtype = num_seqs, chunk, kv_heads, dtype
        self.dim_ld, self.vdim_ld = round8(dim), round8(vdim)
        self.ring_tokens = chunk if max_tokens is None else max(1, min(chunk, max_tokens))
        self.k = torch.zeros((num_seqs, kv_heads, self.ring_tokens, self.dim_ld), dtype=dtype, device=device)
        self.v = torch.zeros((num_seqs, kv_heads, self.ring_tokens, self.vdim_ld), dtype=dtype, device=device)
        self.tickets = torch.zeros(num_seqs * kv_heads * groups, dtype=torch.int32, device=device)   # of the one-token kernel, left zero by it

    def reset(self, slot: int) -> None:
        """Nothing to clear: a row is read only for positions that the sequence itself has written."""

    def tensors(self):
        return [self.k, self.v]

    def gather(self, seq_ids, positions, n_old: int, k: torch.Tensor, v: torch.Tensor, rows_per_seq: int) -> None:
        """The n_old = positions % chunk tokens before `positions` to the first rows of each sequence's block of k / v."""
        from .ops import _dt
        _lib.check(_lib.load().bn_kv_gather(
            self.k.data_ptr(), self.v.data_ptr(), self.ring_tokens, self.chunk, self.kv_heads, self.dim_ld, self.vdim_ld,
            seq_ids.data_ptr(), positions.data_ptr(), seq_ids.numel(), n_old, k.data_ptr(), v.data_ptr(), rows_per_seq,
            _dt(self.dtype), _stream()))


class RecurrentState:
    """What a Mamba-2 layer keeps of a sequence: its state matrices, fp32, and the convolution's last inputs in a ring
    (the input of position p in row p % taps)."""

    def __init__(self, num_seqs: int, heads: int, vdim: int, state: int, channels: int, taps: int, dtype=torch.bfloat16,
                 device="cuda"):
        self.num_seqs = num_seqs
        self.state = torch.zeros((num_seqs, heads, vdim, state), dtype=torch.float32, device=device)
        self.conv = torch.zeros((num_seqs, taps, channels), dtype=dtype, device=device)

    def reset(self, slot: int) -> None:
        self.state[slot].zero_()
        self.conv[slot].zero_()

    def tensors(self):
        return [self.state, self.conv]


class SequenceSlots:
    """Which slot of the per-layer caches and states a live sequence has, and how many tokens it has seen.  A slot that has
    been used is reset in every layer when it is taken again, so what an earlier sequence left never reaches the next one
    (states are made zeroed)."""

    def __init__(self, num_seqs: int, states, device="cuda"):
        self.num_seqs, self.states = num_seqs, list(states)
        self.lens = torch.zeros((num_seqs,), dtype=torch.int32, device=device)
        self.free = list(range(num_seqs - 1, -1, -1))
        self.used = set()

    def acquire(self) -> int:
        if not self.free:
            raise RuntimeError(f"all {self.num_seqs} sequence slots are in use")
        slot = self.free.pop()
        if slot in self.used:
            self.lens[slot] = 0
            for s in self.states:
                s.reset(slot)
        self.used.add(slot)
        return slot

    def release(self, slot: int) -> None:
        if slot in self.free or not 0 <= slot < self.num_seqs:
            raise RuntimeError(f"slot {slot} is not in use")
        self.free.append(slot)

    def tensors(self):
        return [self.lens] + [t for s in self.states for t in s.tensors()]
