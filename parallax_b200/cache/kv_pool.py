"""Device tensors of the paged caches of one pipeline stage.

One cache object per decoder layer, chosen by layer kind (same taxonomy as the reference's
hybrid cache, ``src/parallax/server/cache_manager.py:188-259``):

* ``attention``      K, V            ``[blocks, Hkv, page, D]`` (heads and columns may differ from layer to layer; none
                     for a layer that reads another layer's)
* ``mla_attention``  latent | rope   ``[blocks, 1, page, kv_lora + rope]`` (one tensor; the widths may differ
                     from layer to layer)
* ``dsa_attention``  MLA cache + lightning-indexer keys ``[blocks, 1, page, index_dim]``
* ``linear``         conv state ``[slots, conv_dim, k-1]`` + recurrent state
                     ``[slots, Hv, Dv, Dk]`` (per request slot, not paged)

Any layer may keep per-request slots beside its pages (``ModelConfig.slot_dims``), e.g. the window of a short
convolution in front of softmax attention.

A layer that runs several times for a token (``ModelConfig.layer_passes``) has one cache object per pass; block tables
and slots are the same for all of them.

Layouts are chosen for the sm_100a kernels (whole pages of one head are contiguous), not
for compatibility with the reference's Metal layouts.
"""

from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Optional

import torch

from parallax_b200.models.config import ATTENTION, DSA_ATTENTION, MLA_ATTENTION, MSA_ATTENTION, ModelConfig


@dataclass
class LayerCache:
    kind: str
    k: Optional[torch.Tensor] = None        # attention K / MLA latent+rope
    v: Optional[torch.Tensor] = None        # attention V
    index_k: Optional[torch.Tensor] = None  # DSA / MSA indexer keys
    conv_state: Optional[torch.Tensor] = None
    rec_state: Optional[torch.Tensor] = None
    # e4m3 K / V caches hold value / scale; the attention kernels multiply by the scale again
    k_scale: float = 1.0
    v_scale: float = 1.0
    # a layer that runs several times for a token: the caches of its later passes
    later: list = field(default_factory=list)

    @property
    def passes(self) -> list:
        """The caches of the layer's passes, in order."""
        return [self, *self.later]

    @property
    def kv_scale(self) -> tuple:
        return (self.k_scale, self.v_scale)

    def __iter__(self):  # lets attention layers unpack ``k, v = cache``
        yield self.k
        yield self.v


def kv_cache_torch_dtype(name: Optional[str], model_dtype):
    """Storage dtype of the K / V pages for a ``--kv-cache-dtype`` value."""
    if name in (None, "", "auto"):
        return model_dtype
    if name in ("fp8", "fp8_e4m3", "float8_e4m3fn"):
        return torch.float8_e4m3fn
    if name in ("bf16", "bfloat16"):
        return torch.bfloat16
    raise ValueError(f"unknown KV cache dtype {name!r} (auto, bf16, fp8_e4m3)")


def slot_dims(cfg: ModelConfig, layer: int, tp: int = 1) -> tuple:
    """``ModelConfig.slot_dims`` of one tensor-parallel rank, ``(None, None)`` for a layer without slots."""
    conv, rec = cfg.slot_dims(layer) or (None, None)
    if tp > 1:
        conv = conv and (conv[0] // tp, conv[1])
        rec = rec and (rec[0] // tp, *rec[1:])
    return conv, rec


def bytes_per_block(cfg: ModelConfig, start: int, end: int, page: int, elem: int = 2, tp: int = 1,
                    kv_elem: Optional[int] = None) -> int:
    """``kv_elem``: bytes per element of the K / V pages when they differ from the model's (e4m3: 1)."""
    total = 0
    kv_elem = kv_elem or elem
    for li in range(start, end):
        kind, passes = cfg.layer_kind(li), cfg.layer_passes(li)
        if kind in (ATTENTION, MSA_ATTENTION):
            heads, cols = cfg.kv_dims(li) or (0, 0)
            total += passes * 2 * (heads and max(1, heads // tp)) * page * cols * kv_elem
            if kind == MSA_ATTENTION:
                total += page * int(cfg.raw.get("index_head_dim") or 0) * elem
        elif kind in (MLA_ATTENTION, DSA_ATTENTION):
            total += passes * page * sum(cfg.latent_dims(li)) * elem
            if kind == DSA_ATTENTION:
                total += page * cfg.index_head_dim * elem
    return total


def bytes_per_linear_slot(cfg: ModelConfig, start: int, end: int, elem: int = 2, tp: int = 1) -> int:
    total = 0
    for li in range(start, end):
        conv, rec = slot_dims(cfg, li, tp)
        total += cfg.layer_passes(li) * ((math.prod(conv) * elem if conv else 0) + (math.prod(rec) * 4 if rec else 0))
    return total


class KVPool:
    def __init__(self, cfg: ModelConfig, start_layer: int, end_layer: int, num_blocks: int,
                 page_size: int, device, dtype, tp: int = 1, num_linear_slots: int = 0,
                 kv_cache_dtype: Optional[str] = None, kv_scale: tuple = (1.0, 1.0)):
        """``kv_cache_dtype="fp8_e4m3"`` keeps the K / V pages of the softmax-attention layers as e4m3 bytes
        (half the memory and half the bytes a decode step reads); latent, indexer and recurrent caches stay in
        the model's dtype."""
        kv_dt = kv_cache_torch_dtype(kv_cache_dtype, dtype)
        self.kv_cache_dtype = kv_dt
        self.cfg = cfg
        self.num_blocks = num_blocks
        self.page_size = page_size
        self.device = torch.device(device)
        self.dtype = dtype
        self.layers: list[LayerCache] = []
        for li in range(start_layer, end_layer):
            first, *rest = [self._layer_cache(li, kv_dt, tp, num_linear_slots, kv_scale) for _ in range(cfg.layer_passes(li))]
            first.later = rest
            self.layers.append(first)

    def _layer_cache(self, li: int, kv_dt, tp: int, num_linear_slots: int, kv_scale: tuple) -> LayerCache:
        cfg, num_blocks, page_size, dtype = self.cfg, self.num_blocks, self.page_size, self.dtype
        kind = cfg.layer_kind(li)
        lc = LayerCache(kind)
        if kind in (ATTENTION, MSA_ATTENTION):
            dims = cfg.kv_dims(li)
            if dims is not None:
                shape = (num_blocks, max(1, dims[0] // tp), page_size, dims[1])
                lc.k = torch.zeros(shape, device=self.device, dtype=kv_dt)
                lc.v = torch.zeros(shape, device=self.device, dtype=kv_dt)
            if kv_dt == torch.float8_e4m3fn:
                lc.k_scale, lc.v_scale = float(kv_scale[0]), float(kv_scale[1])
            if kind == MSA_ATTENTION:
                lc.index_k = torch.zeros((num_blocks, 1, page_size, int(cfg.raw.get("index_head_dim") or 0)),
                                         device=self.device, dtype=dtype)
        elif kind in (MLA_ATTENTION, DSA_ATTENTION):
            lc.k = torch.zeros((num_blocks, 1, page_size, sum(cfg.latent_dims(li))),
                               device=self.device, dtype=dtype)
            if kind == DSA_ATTENTION:
                lc.index_k = torch.zeros((num_blocks, 1, page_size, cfg.index_head_dim),
                                         device=self.device, dtype=dtype)
        conv, rec = slot_dims(cfg, li, tp)
        if conv is not None:
            lc.conv_state = torch.zeros((num_linear_slots, *conv), device=self.device, dtype=dtype)
        if rec is not None:
            lc.rec_state = torch.zeros((num_linear_slots, *rec), device=self.device, dtype=torch.float32)
        return lc

    def caches(self):
        """Every cache object of the stage: one per layer and pass."""
        return [c for lc in self.layers for c in lc.passes]

    def zero_slot(self, slot: int) -> None:
        for t in self._slot_tensors():
            t[slot].zero_()

    def copy_slot(self, dst: int, src: int) -> None:
        for t in self._slot_tensors():
            t[dst].copy_(t[src])

    def _slot_tensors(self):
        return [t for lc in self.caches() for t in (lc.conv_state, lc.rec_state) if t is not None]

    def nbytes(self) -> int:
        n = 0
        for lc in self.caches():
            for t in (lc.k, lc.v, lc.index_k, lc.conv_state, lc.rec_state):
                if t is not None:
                    n += t.numel() * t.element_size()
        return n


def plan_num_blocks(cfg: ModelConfig, start: int, end: int, page: int, free_bytes: int,
                    fraction: float, elem: int = 2, tp: int = 1, max_tokens: Optional[int] = None,
                    kv_elem: Optional[int] = None) -> int:
    """Number of KV blocks that fit into ``fraction`` of the free device memory."""
    per_block = bytes_per_block(cfg, start, end, page, elem, tp, kv_elem)
    if per_block == 0:
        return 0
    n = int(free_bytes * fraction) // per_block
    if max_tokens is not None:
        n = min(n, (max_tokens + page - 1) // page)
    return max(n, 0)
