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

Every mixer says what the cache keeps for it: pages (``kv_dims``, one row per token) and / or a slot per
request (``slot_dims``: the last inputs of a short convolution, a recurrent state).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

ACT_SILU, ACT_CLIPPED, ACT_GELU_TANH = 0, 1, 2      # the modes of ops.act_mul / ops.glu_linear


@dataclass(frozen=True)
class RotarySpec:
    """Rotary embedding of the first ``dims`` dimensions, frequencies ``base ** (-2 i / dims)``. Which dimensions
    form a pair (neighbours, or ``i`` and ``i + dims / 2``) is a property of the mixer's kernel."""

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

    kind = "mla_attention"
    kv_from = None
    slot_dims = None

    @property
    def kv_heads(self) -> int:
        return self.heads

    @property
    def q_width(self) -> int:
        return self.dim + self.rot_dim

    @property
    def row_width(self) -> int:
        """Elements per cached token."""
        return self.kv_rank + self.rot_dim


@dataclass(frozen=True)
class AttentionSpec:
    """Softmax attention with grouped heads: a short causal convolution on q, k and v, RMS norm over the whole q and
    k projections, half-split rotation, sinks, an output gate."""

    heads: int
    kv_heads: int
    dim: int            # query / key dimensions per head
    vdim: int           # value dimensions per head
    scale: float
    rot: RotarySpec
    conv: int = 0       # taps of the convolution (0: none)
    kv_from: Optional[int] = None    # layer whose cached keys and values this layer reads instead of its own
    window: int = 0

    kind = "attention"

    @property
    def q_rows(self) -> int:
        return self.heads * self.dim

    @property
    def k_rows(self) -> int:
        return 0 if self.kv_from is not None else self.kv_heads * self.dim

    @property
    def v_rows(self) -> int:
        return 0 if self.kv_from is not None else self.kv_heads * self.vdim

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def head_cols(self) -> int:
        """Columns of a cached key / value row (and of a query): the head size padded with zeros to what the
        tensor-core attention kernels take."""
        d = max(self.dim, self.vdim)
        return 64 if d <= 64 else 128 if d <= 128 else d + -d % 8

    @property
    def kv_dims(self) -> Optional[tuple[int, int]]:
        return None if self.kv_from is not None else (self.kv_heads, self.head_cols)

    @property
    def slot_dims(self) -> Optional[tuple]:
        if self.conv <= 1:
            return None
        return (self.conv - 1, self.q_rows + self.k_rows + self.v_rows), None

    q_width = property(lambda self: self.dim)


@dataclass(frozen=True)
class LightningSpec:
    """Linear attention with a fixed decay per head: ``S <- decay * S + k v^T``, ``o = S^T q``."""

    heads: int
    dim: int
    vdim: int
    decay: tuple

    kind = "linear"
    kv_from = None
    kv_dims = None
    window = 0

    @property
    def kv_heads(self) -> int:
        return self.heads

    @property
    def q_rows(self) -> int:
        return self.heads * self.dim

    k_rows = q_rows

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    v_rows = out_width

    @property
    def slot_dims(self) -> tuple:
        return None, (self.heads, self.dim, self.vdim)

    q_width = property(lambda self: self.dim)


@dataclass(frozen=True)
class ClippedGLUSpec:
    """``down((up' + 1) * g' * sigmoid(alpha g'))``, ``g' = min(gate, limit)``, ``up' = clamp(up, -limit, limit)``."""

    ff: int
    limit: float


@dataclass(frozen=True)
class GLUSpec:
    """``down(act(gate) * up)``."""

    ff: int
    act: int


@dataclass(frozen=True)
class RoutedSpec:
    """Mixture of gated experts. The router's softmax covers ``experts`` experts with weights and ``identity`` ones
    that return their input; ``top`` of them are chosen by score + correction, out of the ``groups_keep`` best of
    ``groups`` groups of neighbours (a group counts as its best expert), and weighted by their scores, normalised."""

    experts: int
    identity: int
    top: int
    expert: GLUSpec
    groups: int = 1
    groups_keep: int = 1
    shared: Optional[GLUSpec] = None    # runs for every token, times a sigmoid gate per token

    @property
    def outputs(self) -> int:
        """Scores per token."""
        return self.experts + self.identity

    @property
    def ff(self) -> int:
        return self.expert.ff


@dataclass(frozen=True)
class BigramSpec:
    """Hashed embedding of (previous token, token): row ``(prev * mul_prev + cur * mul_cur) mod buckets``; a
    sequence's first token uses row ``buckets``."""

    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: object
    mlp: Optional[object]


def _rotary(m: dict, width: int) -> RotarySpec:
    rot = RotarySpec(float(m["rot"]["base"]), int(m["rot"]["dims"]))
    if rot.dims > width or rot.dims % 2:
        raise ValueError(f"rotary dims {rot.dims} do not fit {width} dimensions")
    return rot


def _latent_attention(m: dict) -> LatentAttentionSpec:
    mask = m.get("mask") or {}
    return LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                               kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot=_rotary(m, int(m["rot_dim"])),
                               window=int(mask.get("size") or 0))


def _attention(m: dict) -> AttentionSpec:
    spec = AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                         scale=float(m["scale"]), rot=_rotary(m, int(m["dim"])), conv=int(m.get("conv") or 0),
                         kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
    if spec.heads % spec.kv_heads:
        raise ValueError(f"{spec.heads} query heads cannot share {spec.kv_heads} key / value heads evenly")
    return spec


def _lightning(m: dict) -> LightningSpec:
    spec = LightningSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                         decay=tuple(float(d) for d in m["decay"]))
    if len(spec.decay) != spec.heads:
        raise ValueError(f"{len(spec.decay)} decays for {spec.heads} heads")
    return spec


def _clipped_glu(m: dict) -> ClippedGLUSpec:
    return ClippedGLUSpec(ff=int(m["ff"]), limit=float(m["limit"]))


def _gelu_glu(m: dict) -> GLUSpec:
    return GLUSpec(ff=int(m["ff"]), act=ACT_GELU_TANH)


def _routed(m: dict) -> RoutedSpec:
    r, groups, shared = m["router"], m["router"].get("groups") or {}, m.get("shared")
    spec = RoutedSpec(experts=int(r["experts"]), identity=int(r.get("identity") or 0), top=int(r["top"]),
                      expert=GLUSpec(int(m["expert"]["ff"]), ACT_SILU), groups=int(groups.get("count") or 1),
                      groups_keep=int(groups.get("keep") or 1),
                      shared=None if shared is None else GLUSpec(int(shared["ff"]), ACT_SILU))
    if spec.outputs % spec.groups or not 1 <= spec.groups_keep <= spec.groups:
        raise ValueError(f"{spec.outputs} experts do not form {spec.groups} groups of which {spec.groups_keep} are kept")
    if spec.top > spec.outputs // spec.groups * spec.groups_keep:
        raise ValueError(f"{spec.top} experts per token, but only {spec.groups_keep} groups of "
                         f"{spec.outputs // spec.groups} to choose from")
    return spec


# per architecture: layer types and feed-forward kinds its configs may name
_DESIGNS = {
    "Piburax": ({"latent_attention": _latent_attention}, {"dense": _clipped_glu}),
    "Zudepel": ({"attention": _attention, "lightning": _lightning}, {"dense": _gelu_glu, "moe": _routed}),
}


def parse_layers(architecture: str, entries: list) -> list:
    if architecture not in _DESIGNS:
        raise ValueError(f"no layer-list design {architecture!r}; known: {sorted(_DESIGNS)}")
    mixers, feed_forwards = _DESIGNS[architecture]
    specs = []
    for i, entry in enumerate(entries):
        kind, mlp = entry.get("type"), entry.get("mlp")
        if kind not in mixers:
            raise ValueError(f"unknown layer type {kind!r}; known: {sorted(mixers)}")
        if mlp is not None:
            ff_kind = mlp.get("kind", "dense")
            if ff_kind not in feed_forwards:
                raise ValueError(f"unknown feed-forward kind {ff_kind!r}; known: {sorted(feed_forwards)}")
            mlp = feed_forwards[ff_kind](mlp)
        mixer = mixers[kind](entry["mixer"])
        if mixer.kv_from is not None:
            _check_shared_kv(specs, i, mixer)
        specs.append(LayerSpec(mixer, mlp))
    return specs


def _check_shared_kv(before: list, i: int, m: AttentionSpec) -> None:
    src = before[m.kv_from].mixer if 0 <= m.kv_from < i else None
    if not isinstance(src, AttentionSpec) or src.kv_from is not None:
        raise ValueError(f"layer {i} reads the keys of layer {m.kv_from}, which is no earlier layer with keys of its own")
    if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
        raise ValueError(f"layer {i} and layer {m.kv_from}, whose keys it reads, differ in their key / value heads")


def parse_bigram(emb: dict) -> Optional[BigramSpec]:
    b = emb.get("bigram")
    return None if b is None else BigramSpec(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"]))
