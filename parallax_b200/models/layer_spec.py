"""Per-layer descriptions of models whose ``config.json`` lists its layers one by one.

Most checkpoints describe a decoder with one set of sizes and a few switches
(:class:`parallax_b200.models.config.ModelConfig`). A layer-list config instead gives every layer its
own mixer and feed-forward with their own sizes and constants, so that two layers of one model may
differ in anything. The classes here are the normalised form of such entries; a mixer or feed-forward
kind is one frozen dataclass, and :func:`parse_layer` is the table from config entry to dataclass.

Config layout (``config_from_layer_list``)::

    architecture, vocab, width, norm.eps, residual_mult,
    embedding: {scale, bigram: {buckets, mul_prev, mul_cur} | null},
    layers: [{type, mixer: {...}, mlp: {...} | null}, ...]
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional


@dataclass(frozen=True)
class RotarySpec:
    """Interleaved rotary embedding of the first ``dims`` dimensions, frequencies ``base ** (-2 i / dims)``."""

    base: float
    dims: int


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Latent attention: per token a ``kv_rank``-wide latent and one ``rot_dim``-wide rotated key are cached."""

    heads: int
    dim: int            # unrotated query / key dimensions per head
    rot_dim: int        # rotated query / key dimensions per head
    vdim: int           # value dimensions per head
    kv_rank: int
    scale: float        # factor of the attention scores
    rot: RotarySpec
    window: int = 0     # keys a query sees, itself included (0: all before it)

    @property
    def q_width(self) -> int:
        return self.dim + self.rot_dim

    @property
    def row_width(self) -> int:
        """Elements per cached token."""
        return self.kv_rank + self.rot_dim


@dataclass(frozen=True)
class ClippedGLUSpec:
    """``down((up' + 1) * g' * sigmoid(alpha g'))``, ``g' = min(gate, limit)``, ``up' = clamp(up, -limit, limit)``."""

    ff: int
    limit: float


@dataclass(frozen=True)
class BigramSpec:
    """Hashed embedding of (previous token, token): row ``(prev * mul_prev + cur * mul_cur) mod buckets``; a
    sequence's first token uses row ``buckets``."""

    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentAttentionSpec
    mlp: Optional[ClippedGLUSpec]


def _latent_attention(m: dict) -> LatentAttentionSpec:
    rot = m["rot"]
    mask = m.get("mask") or {}
    spec = LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                               kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                               rot=RotarySpec(float(rot["base"]), int(rot["dims"])), window=int(mask.get("size") or 0))
    if spec.rot.dims > spec.rot_dim or spec.rot.dims % 2:
        raise ValueError(f"rotary dims {spec.rot.dims} do not fit a rotated part of {spec.rot_dim} dimensions")
    return spec


def _clipped_glu(m: dict) -> ClippedGLUSpec:
    return ClippedGLUSpec(ff=int(m["ff"]), limit=float(m["limit"]))


_MIXERS = {"latent_attention": _latent_attention}
_FEED_FORWARDS = {"dense": _clipped_glu}


def parse_layer(entry: dict) -> LayerSpec:
    kind = entry.get("type")
    if kind not in _MIXERS:
        raise ValueError(f"unknown layer type {kind!r}; known: {sorted(_MIXERS)}")
    mlp = entry.get("mlp")
    if mlp is not None:
        if mlp.get("kind", "dense") not in _FEED_FORWARDS:
            raise ValueError(f"unknown feed-forward kind {mlp.get('kind')!r}; known: {sorted(_FEED_FORWARDS)}")
        mlp = _FEED_FORWARDS[mlp.get("kind", "dense")](mlp)
    return LayerSpec(_MIXERS[kind](entry["mixer"]), mlp)


def parse_bigram(emb: dict) -> Optional[BigramSpec]:
    b = emb.get("bigram")
    return None if b is None else BigramSpec(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"]))
