"""Per-layer descriptions of models whose ``config.json`` lists its layers one by one.

Most checkpoints describe a decoder with one set of sizes and a few switches
(:class:`parallax_b200.models.config.ModelConfig`). A layer-list config instead gives every layer its
own mixer and feed-forward with their own sizes and constants, so that two layers of one model may
differ in anything. The classes here are the normalised form of such entries; a mixer or feed-forward
kind is one frozen dataclass, and :func:`parse_layer` is the table from config entry to dataclass.

Config layout (``config_from_layer_list``)::

    architecture, vocab, width, norm: {eps, groups}, residual_mult,
    embedding: {scale, bigram: {buckets, mul_prev, mul_cur} | null},
    loop: {start, stop, times} | null, token_side: {dim} | null,
    layers: [{type, mixer: {...}, mlp: {...} | null}, ...]

Every mixer says what the cache keeps for it: pages (``kv_dims``, one row per token) and / or a slot per
request (``slot_dims``: the last inputs of a short convolution, a recurrent state). A layer inside a loop keeps all of
that once per pass.
"""

from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Optional

# the modes of ops.act_mul / ops.glu_linear / ops.act_linear (the square of relu: act_linear only)
ACT_SILU, ACT_CLIPPED, ACT_GELU_TANH, ACT_RELU_SQUARED = 0, 1, 2, 3


@dataclass(frozen=True)
class RotarySpec:
    """Rotary embedding of the first ``dims`` dimensions, frequencies ``base ** (-2 i / dims)``. Which dimensions
    form a pair (neighbours, or ``i`` and ``i + dims / 2``) is a property of the mixer's kernel."""

    base: float
    dims: int
    scaling: Optional[tuple] = None    # (factor, low, high, original): long wavelengths stretched (rope.stretched_frequencies)


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
    q_rank: int = 0     # width of the normed latent that queries go through (0: projected directly)
    gated: bool = True  # whether the heads are multiplied by sigmoid(W_g x)

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
    """Attention with grouped heads: optionally a short causal convolution on q, k and v and RMS norm over the
    whole q and k projections, or a norm without weights over each head; half-split rotation, an output gate. With a
    ``window`` a query sees that many keys, itself included, and the sequence's first ``keep_first`` ones. The weights of
    the visible keys are a softmax of the scores (optionally soft-capped), or sigmoids that nothing normalises."""

    heads: int
    kv_heads: int
    dim: int            # query / key dimensions per head
    vdim: int           # value dimensions per head
    scale: float
    rot: Optional[RotarySpec]
    conv: int = 0       # taps of the convolution (0: none)
    kv_from: Optional[int] = None    # layer whose cached keys and values this layer reads instead of its own
    window: int = 0
    keep_first: int = 0
    softcap: float = 0.0             # scores: softcap * tanh(score / softcap) (0: none)
    sigmoid: bool = False            # weights: sigmoid(score + a number per head)
    q_temp: Optional[tuple] = None   # (coef, every): queries times 1 + coef ln(floor((p + 1) / every) + 1) at position p
    v_mix: bool = False              # values are mixed with those of the first layer that mixes them
    v_first: Optional[int] = None    # that layer (None: it is this one, or nothing is mixed)

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
class MatrixMemorySpec:
    """mLSTM: linear attention whose decay and input weight are gates of the token (exponential, soft-capped logarithms
    kept stable by a running maximum), with a normaliser beside the state."""

    heads: int
    dim: int
    vdim: int
    gate_cap: float

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
        return None, (self.heads, memory_words(self.dim, self.vdim))

    q_width = property(lambda self: self.dim)


MEMORY_SLICE = 32    # value columns that share one copy of a matrix memory's normaliser and maximum


def memory_words(dim: int, vdim: int) -> int:
    """fp32 words of one head's matrix memory in a state slot: the matrix ``[dim, vdim]``, then for every slice of
    :data:`MEMORY_SLICE` value columns a copy of the normaliser ``[dim]``, then their maxima; padded to 16 bytes. (Every
    thread block owns whole slices with their copies, so the blocks of a head never wait for one another.)"""
    slices = -(-vdim // MEMORY_SLICE)
    n = dim * vdim + slices * (dim + 1)
    return n + -n % 4


def _up8(n: int) -> int:
    return n + -n % 8


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule with a decay per key channel, behind short convolutions: ``S <- g S``, ``u = beta (v - S^T k)``,
    ``S <- S + k u^T``, ``o = S^T q``; q and k are unit vectors, shared by neighbouring heads."""

    heads: int
    kv_heads: int       # heads of q and k
    dim: int
    vdim: int
    conv: int           # taps of the convolutions on q, k and v

    kind = "linear"
    kv_from = None
    kv_dims = None
    window = 0

    @property
    def q_rows(self) -> int:
        return self.kv_heads * self.dim

    k_rows = q_rows

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    v_rows = out_width

    @property
    def channels(self) -> int:
        """Convolved channels q | k | v, each part padded to a multiple of 8."""
        return 2 * _up8(self.q_rows) + _up8(self.v_rows)

    @property
    def slot_dims(self) -> tuple:
        return (self.conv - 1, self.channels) if self.conv > 1 else None, (self.heads, self.dim, self.vdim)

    q_width = property(lambda self: self.dim)


@dataclass(frozen=True)
class StateSpaceSpec:
    """Mamba-2: ``S <- exp(-a dt) S + dt B x^T``, ``y = S^T C + D x`` per head; B and C are shared by the heads of a group
    and, like x, pass a short convolution. The gate comes before a norm over ``norm_groups`` parts of the heads."""

    heads: int
    groups: int
    state: int
    vdim: int
    conv: int
    norm_groups: int

    kind = "linear"
    kv_from = None
    kv_dims = None
    window = 0
    kv_heads = property(lambda self: self.groups)
    q_width = property(lambda self: self.state)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def bc_rows(self) -> int:
        return self.groups * self.state

    @property
    def channels(self) -> int:
        """Convolved channels x | B | C, each part padded to a multiple of 8."""
        return _up8(self.out_width) + 2 * _up8(self.bc_rows)

    @property
    def slot_dims(self) -> tuple:
        return (self.conv - 1, self.channels) if self.conv > 1 else None, (self.heads, self.state, self.vdim)


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers that read the same input: attention with pages beside a recurrent memory with a slot, added with fixed
    factors; ``normed``: each output is RMS-normed over the model width first."""

    left: AttentionSpec
    right: object
    left_scale: float
    right_scale: float
    normed: bool = False

    kind = "attention"
    kv_from = None

    heads = property(lambda self: self.left.heads)
    kv_heads = property(lambda self: self.left.kv_heads)
    vdim = property(lambda self: max(self.left.vdim, self.right.vdim))
    rot = property(lambda self: self.left.rot)
    window = property(lambda self: self.left.window)
    kv_dims = property(lambda self: self.left.kv_dims)
    slot_dims = property(lambda self: self.right.slot_dims)
    q_width = property(lambda self: self.left.q_width)


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
class DenseSpec:
    """``down(act(up))``."""

    ff: int
    act: int


@dataclass(frozen=True)
class RoutedSpec:
    """Mixture of gated experts. The router's scores (softmax or sigmoid) cover ``experts`` experts with weights and
    ``identity`` ones that return their input; ``top`` of them are chosen by score (+ correction), out of the
    ``groups_keep`` best of ``groups`` groups of neighbours (a group counts as its best expert), and weighted by their
    scores, normalised or not. The weight multiplies an expert's output, or its input."""

    experts: int
    identity: int
    top: int
    expert: object      # GLUSpec or ClippedGLUSpec
    groups: int = 1
    groups_keep: int = 1
    shared: Optional[GLUSpec] = None    # runs for every token
    shared_gate: bool = True            # times a sigmoid gate per token
    sigmoid: bool = False               # scores: sigmoid instead of softmax
    correction: bool = True             # a learned number per expert takes part in the choice
    normalised: bool = True
    weighted_input: bool = False
    bias: bool = False                  # a learned number per expert is part of its logit

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
class LoopSpec:
    """Layers ``start .. stop - 1`` run ``times`` times in a row with the same weights, each pass with a cache and state of
    its own."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: object
    mlp: Optional[object]


def _rotary(m: dict, width: int) -> RotarySpec:
    s = m["rot"].get("scaling")
    scaling = None if s is None else tuple(float(s[n]) for n in ("factor", "low", "high", "original"))
    rot = RotarySpec(float(m["rot"]["base"]), int(m["rot"]["dims"]), scaling)
    if scaling is not None and not (scaling[0] > 0 and scaling[2] > scaling[1]):
        raise ValueError(f"rotary scaling {s} stretches nothing")
    if rot.dims > width or rot.dims % 2:
        raise ValueError(f"rotary dims {rot.dims} do not fit {width} dimensions")
    return rot


def _latent_attention(m: dict) -> LatentAttentionSpec:
    mask = m.get("mask") or {}
    return LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                               kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot=_rotary(m, int(m["rot_dim"])),
                               window=int(mask.get("size") or 0))


def _query_latent_attention(m: dict) -> LatentAttentionSpec:
    return replace(_latent_attention(m), q_rank=int(m["q_rank"]), gated=False)


def _attention(m: dict) -> AttentionSpec:
    spec = AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                         scale=float(m["scale"]), rot=_rotary(m, int(m["dim"])) if m.get("rot") else None,
                         conv=int(m.get("conv") or 0),
                         kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
    if spec.heads % spec.kv_heads:
        raise ValueError(f"{spec.heads} query heads cannot share {spec.kv_heads} key / value heads evenly")
    return spec


def _windowed_attention(m: dict) -> AttentionSpec:
    mask = m.get("mask") or {}
    return replace(_attention(m), window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0))


def _lightning(m: dict) -> LightningSpec:
    spec = LightningSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                         decay=tuple(float(d) for d in m["decay"]))
    if len(spec.decay) != spec.heads:
        raise ValueError(f"{len(spec.decay)} decays for {spec.heads} heads")
    return spec


def _memory(m: dict) -> MatrixMemorySpec:
    spec = MatrixMemorySpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))
    if spec.gate_cap <= 0:
        raise ValueError(f"a gate cap of {spec.gate_cap} closes every gate")
    return spec


def _parallel(m: dict) -> ParallelSpec:
    return ParallelSpec(left=_windowed_attention(m["left"]), right=_memory(m["right"]), left_scale=float(m["left_scale"]),
                        right_scale=float(m["right_scale"]))


def _capped_attention(m: dict) -> AttentionSpec:
    return replace(_attention(m), softcap=float(m.get("softcap") or 0), v_mix=bool(m.get("v_mix")))


def _sigmoid_attention(m: dict) -> AttentionSpec:
    t = m.get("q_temp")
    return replace(_attention(m), sigmoid=True, q_temp=None if t is None else (float(t["coef"]), float(t["every"])))


def _delta(m: dict) -> DeltaSpec:
    spec = DeltaSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                     conv=int(m["conv"]))
    if spec.heads % spec.kv_heads or spec.conv < 1:
        raise ValueError(f"{spec.heads} heads, {spec.kv_heads} of q and k, {spec.conv} taps: no delta rule")
    return spec


def _normed_parallel(m: dict) -> ParallelSpec:
    return ParallelSpec(left=_sigmoid_attention(m["left"]), right=_delta(m["right"]), left_scale=0.5, right_scale=0.5, normed=True)


def _state_space(m: dict) -> StateSpaceSpec:
    spec = StateSpaceSpec(heads=int(m["heads"]), groups=int(m["groups"]), state=int(m["state"]), vdim=int(m["vdim"]),
                          conv=int(m["conv"]), norm_groups=int(m["norm_groups"]))
    if spec.heads % spec.groups or spec.out_width % spec.norm_groups or spec.conv < 1:
        raise ValueError(f"{spec.heads} heads of {spec.vdim} in {spec.groups} groups, {spec.norm_groups} parts of the norm, "
                         f"{spec.conv} taps: no state-space mixer")
    return spec


def _clipped_glu(m: dict) -> ClippedGLUSpec:
    return ClippedGLUSpec(ff=int(m["ff"]), limit=float(m["limit"]))


def _gelu_glu(m: dict) -> GLUSpec:
    return GLUSpec(ff=int(m["ff"]), act=ACT_GELU_TANH)


def _relu_squared(m: dict) -> DenseSpec:
    return DenseSpec(ff=int(m["ff"]), act=ACT_RELU_SQUARED)


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


def _sigmoid_routed(m: dict) -> RoutedSpec:
    return replace(_routed(m), sigmoid=True, correction=False, normalised=False, shared_gate=False, weighted_input=True)


def _biased_routed(m: dict) -> RoutedSpec:
    spec = replace(_routed(m), correction=False, shared_gate=False, bias=True, expert=_clipped_glu(m["expert"]))
    if spec.identity or spec.shared or spec.groups > 1:
        raise ValueError("identity experts, a shared expert or groups of experts are not part of this feed-forward")
    return spec


# architectures whose output head is the embedding table
TIED = frozenset({"Kikurax"})

# per architecture: layer types and feed-forward kinds its configs may name
_DESIGNS = {
    "Piburax": ({"latent_attention": _latent_attention}, {"dense": _clipped_glu}),
    "Zudepel": ({"attention": _attention, "lightning": _lightning}, {"dense": _gelu_glu, "moe": _routed}),
    "Zasalix": ({"latent_attention": _query_latent_attention, "parallel": _parallel, "mlstm": _memory},
                {"dense": _relu_squared, "moe": _sigmoid_routed}),
    "Kikurax": ({"parallel": _normed_parallel, "mamba2": _state_space, "attention": _capped_attention}, {"moe": _biased_routed}),
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
        specs.append(LayerSpec(_with_first_values(specs, i, mixer), mlp))
    return specs


def _with_first_values(before: list, i: int, m):
    """The mixer with the index of the first layer that mixes values, where it mixes that layer's."""
    if not getattr(m, "v_mix", False):
        return m
    first = next((j for j, s in enumerate(before) if getattr(s.mixer, "v_mix", False)), None)
    if first is None:
        return m
    src = before[first].mixer
    if src.v_rows != m.v_rows:
        raise ValueError(f"layer {i} and layer {first}, whose values it mixes in, differ in the width of their value heads")
    return replace(m, v_first=first)


def _check_shared_kv(before: list, i: int, m: AttentionSpec) -> None:
    src = before[m.kv_from].mixer if 0 <= m.kv_from < i else None
    if not isinstance(src, AttentionSpec) or src.kv_from is not None:
        raise ValueError(f"layer {i} reads the keys of layer {m.kv_from}, which is no earlier layer with keys of its own")
    if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
        raise ValueError(f"layer {i} and layer {m.kv_from}, whose keys it reads, differ in their key / value heads")


def parse_bigram(emb: dict) -> Optional[BigramSpec]:
    b = emb.get("bigram")
    return None if b is None else BigramSpec(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"]))


def parse_loop(loop: Optional[dict], layers: int) -> Optional[LoopSpec]:
    if not loop:
        return None
    spec = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
    if not 0 <= spec.start < spec.stop <= layers or spec.times < 1:
        raise ValueError(f"layers {spec.start} to {spec.stop - 1}, {spec.times} times, is no loop over {layers} layers")
    return spec
