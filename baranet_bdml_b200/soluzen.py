"""Soluzen: a decoder whose layers are latent attention with a sliding window or Mamba-2, in any order, some of them run
several times in a row with the same weights; every layer also receives an input that depends on the token alone.

This module holds what is particular to the design: how its config.json is read and how its layers are strung together.
The sublayers are in mixers.py, caches and states in kv_cache.py, generation in model.py."""
from __future__ import annotations

import warnings
from dataclasses import dataclass
from typing import List, Optional, Sequence

import torch

from . import ops
from .checkpoint import Weights
from .mixers import GatedMLP, LatentAttention, LatentAttentionConfig, Mamba2Config, Mamba2Mixer, TokenSide
from .model import SequenceLM
from .ops import Pending, round8

MIXERS = {"latent_attention": LatentAttention, "mamba2": Mamba2Mixer}
ACTIVATION = "gelu_tanh"          # of the feed-forward and of the token input


def _mixer_config(kind: str, m: dict):
    if kind == "latent_attention":
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError("latent attention rotates the whole rotated part: rot.dims must equal rot_dim")
        return LatentAttentionConfig(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=m["q_rank"],
                                     kv_rank=m["kv_rank"], window=m["mask"]["size"], rope_base=float(m["rot"]["base"]),
                                     scale=float(m["scale"]))
    if kind == "mamba2":
        return Mamba2Config(heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"], taps=m["conv"],
                            norm_groups=m["norm_groups"])
    raise ValueError(f"unknown mixer {kind!r}")


@dataclass(frozen=True)
class LayerConfig:
    kind: str
    mixer: object
    ff: Optional[int]             # None: the layer has no feed-forward


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class SoluzenConfig:
    vocab_size: int
    width: int
    eps: float
    side_dim: int
    layers: Sequence[LayerConfig]
    loop: Optional[LoopConfig]
    eos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, c: dict) -> "SoluzenConfig":
        layers = []
        for entry in c["layers"]:
            mlp = entry["mlp"]
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerConfig(entry["type"], _mixer_config(entry["type"], entry["mixer"]), None if mlp is None else mlp["ff"]))
        loop = c.get("loop")
        if loop is not None:
            loop = LoopConfig(loop["start"], loop["stop"], loop["times"])
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ValueError(f"bad loop {loop}")
        return cls(vocab_size=c["vocab"], width=c["width"], eps=float(c["norm"]["eps"]), side_dim=c["token_side"]["dim"],
                   layers=tuple(layers), loop=loop)

    def runs(self):
        """(layer, number of the pass that begins with this run or None), in order."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        a, b, times = self.loop.start, self.loop.stop, self.loop.times
        return ([(i, None) for i in range(a)] + [(i, t if i == a else None) for t in range(times) for i in range(a, b)] +
                [(i, None) for i in range(b, n)])


class SoluzenLayer:
    def __init__(self, cfg: LayerConfig, name: str, model: SoluzenConfig, w: Weights, dtype):
        def norm(which):
            return ops.NormWeight(w(f"{name}.{which}", model.width), w(f"{name}.{which}.b", model.width), model.eps)

        def part(prefix):
            return lambda key, *shape: w(f"{name}.{prefix}.{key}", *shape)

        self.norm1 = norm("norm1")
        self.mixer = MIXERS[cfg.kind](cfg.mixer, model.width, model.eps, part("mix"), dtype)
        self.norm2 = self.mlp = None
        if cfg.ff is not None:
            self.norm2, self.mlp = norm("norm2"), GatedMLP(cfg.ff, model.width, ACTIVATION, part("mlp"), dtype)
        self.side = TokenSide(model.side_dim, model.width, model.eps, ACTIVATION, part("side"), dtype)


class SoluzenModel(SequenceLM):
    """The residual stream is fp32 in both dtypes; what reads it is normalised or rounded by the launch that adds the
    sublayer before it (ops.residual_norm)."""

    def __init__(self, config: SoluzenConfig, weights: Weights, dtype=torch.bfloat16):
        super().__init__(config, dtype)
        c, w = config, weights
        n, width, w8 = len(c.layers), c.width, round8(c.width)
        self.embed_tokens = w("embed", c.vocab_size, width).to(device="cuda", dtype=dtype).contiguous()
        # each layer's part of the token input starts on a 16-byte boundary
        self.side8 = round8(c.side_dim)
        side = torch.zeros((c.vocab_size, n, self.side8), dtype=dtype, device="cuda")
        side[:, :, :c.side_dim] = w("side.embed", c.vocab_size, n * c.side_dim).to("cuda").view(c.vocab_size, n, c.side_dim)
        self.side_embed = side.view(c.vocab_size, n * self.side8)
        self.layers = [SoluzenLayer(lc, f"l{i}", c, w, dtype) for i, lc in enumerate(c.layers)]
        self.runs = c.runs()
        if c.loop is not None:
            # the pass input [x; embedding]: in bf16 the stream goes in as its rounding and that rounding's remainder, so
            # that the product reads it with fp32's precision, near enough
            w_in = w("loop.in", width, 2 * width)
            parts = [w_in[:, :width], w_in[:, :width], w_in[:, width:]] if dtype == torch.bfloat16 else [w_in[:, :width], w_in[:, width:]]
            cat = torch.zeros((width, len(parts) * w8), dtype=w_in.dtype)
            for k, p in enumerate(parts):
                cat[:, k * w8:k * w8 + width] = p
            self.loop_in = ops.Linear(cat, dtype)
            self.loop_step = w("loop.step", c.loop.times, width).to(device="cuda", dtype=torch.float32).contiguous()
        self.final_norm = ops.NormWeight(w("final.norm", width), w("final.norm.b", width), c.eps)
        self.head = ops.Linear(w("head", c.vocab_size, width), dtype)
        if w.leftover():
            warnings.warn(f"checkpoint tensors that this design does not have: {w.leftover()[:5]}")

    # ------------------------------------------------------------------ sequences
    def new_states(self, num_seqs: int, max_tokens: Optional[int]):
        """One per layer run, so each pass of the loop has its own; their size does not depend on a sequence's length."""
        return [self.layers[i].mixer.new_state(num_seqs) for i, _ in self.runs]

    # -------------------------------------------------------------------- forward
    def _embed(self, ids: torch.Tensor):
        """(fp32 stream, token inputs of all layers, the pass-input buffer with the embedding in its last part)"""
        c, rows, w8 = self.config, ids.numel(), round8(self.config.width)
        x = torch.empty((rows, c.width), dtype=torch.float32, device="cuda")
        side = torch.empty((rows, self.side_embed.shape[1]), dtype=self.dtype, device="cuda")
        bf16 = self.dtype == torch.bfloat16
        cat = x0 = None
        if c.loop is not None:
            cat = (torch.empty if w8 == c.width else torch.zeros)((rows, self.loop_in.k), dtype=self.dtype, device="cuda")
            x0 = cat[:, self.loop_in.k - w8:]
        ops.embedding_rows(self.embed_tokens, ids, out_f32=x, out_bf16=x0 if bf16 else None, error_word=self._id_error)
        if x0 is not None and not bf16:
            x0[:, :c.width] = x
        if bf16:
            ops.embedding_rows(self.side_embed, ids, out_bf16=side)
        else:
            ops.embedding_rows(self.side_embed, ids, out_f32=side)
        return x, side, cat

    def _forward(self, ids: torch.Tensor, B: int, S: int, seq_ids, positions, n_old: Optional[int]):
        """All layers over B x S new tokens: (the residual stream, its last addend, still pending)."""
        c, dt, width, w8, s8 = self.config, self.dtype, self.config.width, round8(self.config.width), self.side8
        x, side, cat = self._embed(ids)
        pending, row = None, None
        for (i, start_of_pass), state in zip(self.runs, self.states):
            layer = self.layers[i]
            if start_of_pass is not None:
                ops.residual_norm(x, pending, dt, width, keep_sum=False, cast=cat, lo_offset=w8 if dt == torch.bfloat16 else 0)
                x, pending, row = None, Pending(self.loop_in(cat, f32_out=True)), self.loop_step[start_of_pass]
            x, h = ops.residual_norm(x, pending, dt, width, row=row, norm=layer.norm1)
            row = None
            delta = layer.mixer(h, B, S, state, seq_ids, positions, n_old)
            if layer.mlp is not None:
                x, h = ops.residual_norm(x, Pending(delta), dt, width, norm=layer.norm2)
                delta = layer.mlp(h)
            xb = (torch.empty if w8 == width else torch.zeros)((B * S, w8), dtype=dt, device="cuda")
            x, _ = ops.residual_norm(x, Pending(delta), dt, width, cast=xb)
            pending = layer.side(xb, side[:, i * s8:(i + 1) * s8])
        return x, pending

    def _select(self, state, rows: torch.Tensor):
        x, pending = state
        return x.index_select(0, rows), pending.select(rows)

    def _logits(self, state) -> torch.Tensor:
        x, pending = state
        _, h = ops.residual_norm(x, pending, self.dtype, self.config.width, norm=self.final_norm, keep_sum=False)
        return self.head(h, f32_out=True)[:, :self.config.vocab_size]

    def parameters(self) -> List[torch.Tensor]:
        return ops.tensors_of([self.embed_tokens, self.side_embed, self.layers, getattr(self, "loop_in", None),
                               getattr(self, "loop_step", None), self.final_norm, self.head])
