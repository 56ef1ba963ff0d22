"""Duponex: a decoder of grouped-query attention in chunks and squared-ReLU feed-forwards over a residual that is kept as
several streams (hyper-connections): every sublayer reads a weighted sum of them and writes back through a small matrix.  The
attention layers' values are mixed with those of the first layer that takes part in it.

This module holds what is particular to the design: how its config.json is read and how its layers are strung together.
The sublayers are in mixers.py, caches in kv_cache.py, sequences and generation in model.py, the streams in ops.hyper_norm."""
from __future__ import annotations

import warnings
from dataclasses import dataclass
from typing import List, Optional, Sequence

import torch

from . import ops
from .checkpoint import Weights
from .mixers import MLP, ChunkedAttention, ChunkedAttentionConfig
from .model import SequenceLM

ACTIVATION = "relu2"              # of the feed-forward


@dataclass(frozen=True)
class LayerConfig:
    mixer: ChunkedAttentionConfig
    ff: Optional[int]             # None: the layer has no feed-forward


@dataclass(frozen=True)
class DuponexConfig:
    vocab_size: int
    width: int
    eps: float
    streams: int
    embedding_scale: float
    residual_mult: float
    layers: Sequence[LayerConfig]
    eos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, c: dict) -> "DuponexConfig":
        layers = []
        for entry in c["layers"]:
            m, mlp = entry["mixer"], entry.get("mlp")
            if entry["type"] != "attention":
                raise ValueError(f"unknown mixer {entry['type']!r}")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerConfig(
                ChunkedAttentionConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], chunk=m["mask"]["size"],
                                       scale=float(m["scale"]), mixes_values=bool(m.get("v_mix", False))),
                None if mlp is None else mlp["ff"]))
        if c["streams"] < 1:
            raise ValueError(f"streams must be positive, not {c['streams']}")
        if len({(lc.mixer.kv_heads, lc.mixer.vdim) for lc in layers if lc.mixer.mixes_values}) > 1:
            raise ValueError("layers that mix values must agree in key/value heads and value size")
        return cls(vocab_size=c["vocab"], width=c["width"], eps=float(c["norm"]["eps"]), streams=c["streams"],
                   embedding_scale=float(c["embedding"]["scale"]), residual_mult=float(c["residual_mult"]), layers=tuple(layers))


class Sublayer:
    """What surrounds a mixer or a feed-forward: the weights of the sum it reads, the norm of that sum, the scale of its
    result, and how the streams take it up."""

    def __init__(self, name: str, which: int, c: DuponexConfig, w: Weights):
        s = c.streams
        floats = lambda key, *shape: w(f"{name}.hc{which}.{key}", *shape).double().tolist()     # noqa: E731
        self.read, self.mix = floats("in", s), floats("mix", s, s)                             # mix[from][to]
        self.write = [c.residual_mult * v for v in floats("out", s)]
        self.norm = ops.NormWeight(w(f"{name}.norm{which}", c.width), None, c.eps)
        self.scale = w(f"{name}.ls{which}", c.width).to(device="cuda", dtype=torch.float32).contiguous()


class DuponexLayer:
    def __init__(self, cfg: LayerConfig, name: str, model: DuponexConfig, w: Weights, dtype):
        def part(prefix):
            return lambda key, *shape: w(f"{name}.{prefix}.{key}", *shape)

        self.sub1, self.mixer = Sublayer(name, 1, model, w), ChunkedAttention(cfg.mixer, model.width, model.eps, part("mix"), dtype)
        self.sub2 = self.mlp = None
        if cfg.ff is not None:
            self.sub2, self.mlp = Sublayer(name, 2, model, w), MLP(cfg.ff, model.width, ACTIVATION, part("mlp"), dtype)


class DuponexModel(SequenceLM):
    """The streams are fp32 in both dtypes; one launch takes a sublayer's output into them and norms what the next one reads."""

    def __init__(self, config: DuponexConfig, weights: Weights, dtype=torch.bfloat16):
        super().__init__(config, dtype)
        c, w = config, weights
        self.embed_tokens = w("embed", c.vocab_size, c.width).to(device="cuda", dtype=dtype).contiguous()
        self.layers = [DuponexLayer(lc, f"l{i}", c, w, dtype) for i, lc in enumerate(c.layers)]
        self.final_norm = ops.NormWeight(w("final.norm", c.width), None, c.eps)
        self.head = ops.Linear(w("head", c.vocab_size, c.width), dtype)
        self.first_mixing = next((i for i, lc in enumerate(c.layers) if lc.mixer.mixes_values), None)
        subs = [s for layer in self.layers for s in (layer.sub1, layer.sub2) if s is not None]
        # step k leads from the streams before sublayer k - 1's result to what sublayer k reads; the first two find the
        # embedding alone, of which every stream is a copy, and the last one only needs the sum of the streams
        one, n = [1.0], c.streams
        self.steps = [ops.StreamMix([[c.embedding_scale]], [0.0], [sum(subs[0].read)] if subs else [float(n)], keep=False)]
        for k, sub in enumerate(subs):
            mix = sub.mix if k else [[c.embedding_scale * sum(row[t] for row in sub.mix) for t in range(n)]]
            last = k + 1 == len(subs)
            self.steps.append(ops.StreamMix(mix, sub.write, one * n if last else subs[k + 1].read, keep=not last))
        if w.leftover():
            warnings.warn(f"checkpoint tensors that this design does not have: {w.leftover()[:5]}")

    def new_states(self, num_seqs: int, max_tokens: Optional[int]):
        return [layer.mixer.new_state(num_seqs, max_tokens) for layer in self.layers]

    # -------------------------------------------------------------------- forward
    def _forward(self, ids: torch.Tensor, B: int, S: int, seq_ids, positions, n_old: Optional[int]):
        """All layers over B x S new tokens: (streams, the last sublayer's output and its scale, still pending)."""
        c, dt = self.config, self.dtype
        x = torch.empty((B * S, 1, c.width), dtype=torch.float32, device="cuda")
        ops.embedding_rows(self.embed_tokens, ids, out_f32=x.view(B * S, c.width), error_word=self._id_error)
        delta = scale = v_first = None
        steps = iter(self.steps)

        def read(sub):
            """takes the pending output into the streams and norms what `sub` reads"""
            nonlocal x
            new, h = ops.hyper_norm(x, next(steps), dt, sub.norm, delta=delta, delta_scale=scale)
            x = x if new is None else new
            return h

        for i, (layer, state) in enumerate(zip(self.layers, self.states)):
            proj = layer.mixer.project(read(layer.sub1))
            mixed = v_first if layer.mixer.cfg.mixes_values else None
            delta = layer.mixer(proj, B, S, state, seq_ids, positions, n_old, mixed)
            scale = layer.sub1.scale
            if i == self.first_mixing:
                v_first = layer.mixer.values(proj)
            if layer.mlp is not None:
                delta, scale = layer.mlp(read(layer.sub2)), layer.sub2.scale
        return x, delta, scale

    def _select(self, state, rows: torch.Tensor):
        x, delta, scale = state
        return x.index_select(0, rows), delta if delta is None else delta.index_select(0, rows), scale

    def _logits(self, state) -> torch.Tensor:
        x, delta, scale = state
        _, h = ops.hyper_norm(x, self.steps[-1], self.dtype, self.final_norm, delta=delta, delta_scale=scale)
        return self.head(h, f32_out=True)[:, :self.config.vocab_size]

    def parameters(self) -> List[torch.Tensor]:
        return ops.tensors_of([self.embed_tokens, self.layers, self.final_norm, self.head])
