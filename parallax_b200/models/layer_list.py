"""Shared half of the stages whose config lists its layers one by one (:mod:`parallax_b200.models.layer_spec`):
flat checkpoint names (``embed``, ``l<i>.*``, ``final.norm``, ``head``) with shape checks, random weights, refit, an
fp32 residual, and the output head. A family adds its layers: ``weight_shapes``, ``_load_layer`` and
``forward_layers``.

The stages run in bf16 (tensor cores; fp32 where the design keeps fp32) or entirely in fp32
(``dtype=torch.float32``)."""

from __future__ import annotations

import re
from typing import Optional

import torch

from parallax_b200 import ops
from parallax_b200.engine.batch import ForwardBatch
from parallax_b200.models.config import ModelConfig
from parallax_b200.models.decoder import DecoderStage
from parallax_b200.models.layer_spec import RotarySpec
from parallax_b200.models.rope import stretched_frequencies


def pad_rows(w: torch.Tensor, multiple: int) -> torch.Tensor:
    extra = -w.shape[0] % multiple
    if not extra:
        return w.contiguous()
    return torch.cat([w, w.new_zeros((extra,) + tuple(w.shape[1:]))], 0).contiguous()


class ListedLayer:
    """Weights of one layer; subclasses name them in ``__slots__``."""

    __slots__ = ("spec", "layer_idx", "cos_sin")

    def __init__(self):
        for c in type(self).__mro__:
            for s in getattr(c, "__slots__", ()):
                setattr(self, s, None)

    def tensors(self) -> list:
        out = []
        for c in type(self).__mro__:
            for s in getattr(c, "__slots__", ()):
                v = getattr(self, s)
                if isinstance(v, torch.Tensor) and s != "cos_sin":
                    out.append(v)
                elif hasattr(v, "tensors"):
                    out += v.tensors()
        return out


class LayerListStage(DecoderStage):
    _LAYER_KEY = re.compile(r"(?:^|\.)l(\d+)\.")
    _GLOBAL_KEYS = ("embed", "bigram", "final.norm", "head")
    _GLOBAL_TENSORS = ("embed", "bigram", "norm_w", "lm_head")
    layer_class = ListedLayer
    final_norm = ops.NORM_LAYER

    def __init__(self, cfg: ModelConfig, start_layer: int, end_layer: int, device, dtype=None,
                 max_positions: Optional[int] = None):
        super().__init__(cfg, start_layer, end_layer, device, dtype, max_positions)
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"{cfg.architecture} runs in bfloat16 or float32, not {self.dtype}")
        del self.lora                   # no per-request adapters for these families (checked with hasattr)
        self.bigram: Optional[torch.Tensor] = None
        self.layers = [self.layer_class() for _ in range(start_layer, end_layer)]
        self.cos_sin = None             # tables are per layer: base and width are
        self._tables: dict[RotarySpec, torch.Tensor] = {}
        for gi, lw in enumerate(self.layers, start_layer):
            self._describe(lw, gi)

    @property
    def hidden_dtype(self) -> torch.dtype:
        return torch.float32

    def _describe(self, lw: ListedLayer, gi: int) -> None:
        lw.layer_idx, lw.spec = gi, self.cfg.layer_specs[gi]
        rot = getattr(lw.spec.mixer, "rot", None)
        if rot is None:
            return
        if rot not in self._tables:
            inv = rot.base ** (-torch.arange(0, rot.dims, 2, dtype=torch.float64) / rot.dims)
            if rot.scaling is not None:
                inv = stretched_frequencies(inv, *rot.scaling)
            self._tables[rot] = ops.build_cos_sin(self.max_positions, rot.dims, rot.base, device=self.device, inv_freq=inv)
        lw.cos_sin = self._tables[rot]

    # ------------------------------------------------------------------ weights
    def global_shapes(self) -> dict[str, tuple]:
        """Checkpoint tensors outside the layers that this stage holds (name -> shape)."""
        cfg, W, sh = self.cfg, self.cfg.hidden_size, {}
        if self.is_first or (self.is_last and cfg.tie_word_embeddings):
            sh["embed"] = (cfg.vocab_size, W)
        if self.is_first and cfg.bigram is not None:
            sh["bigram"] = (cfg.bigram.buckets + 1, W)
        if self.is_last:
            sh["final.norm"] = (W,)
            if not cfg.tie_word_embeddings:
                sh["head"] = (cfg.vocab_size, W)
        return sh

    def weight_shapes(self, gi: int) -> dict[str, tuple]:
        """Checkpoint tensors of layer ``gi`` (name -> shape; -1: a size that only the tensor itself gives)."""
        raise NotImplementedError

    def _load_layer(self, lw: ListedLayer, gi: int, tensors) -> None:
        raise NotImplementedError

    def init_random(self, seed: int = 0, std: float = 0.02) -> None:
        cfg, dev = self.cfg, self.device
        g = torch.Generator(device=dev)

        def rnd(shape, k):
            g.manual_seed(seed * 1000003 + k)
            return (torch.randn(*shape, generator=g, device=dev, dtype=torch.float32) * std).to(torch.bfloat16)

        seeds = {"embed": 900001, "head": 900002, "bigram": 900003, "side.embed": 900004, "loop.step": 900005}
        self._load_globals({name: self._random(name, shape, lambda s, k=seeds.get(name): rnd(s, k))     # (alike on every stage)
                            for name, shape in self.global_shapes().items()})
        for gi, lw in enumerate(self.layers, self.start_layer):      # layer by layer: one raw copy at a time
            layer = {name: self._random(name, shape, lambda s, i=i: rnd(s, gi * 4096 + i))
                     for i, (name, shape) in enumerate(self.weight_shapes(gi).items())}
            self._load_layer(lw, gi, layer)

    def _random(self, name: str, shape: tuple, rnd) -> torch.Tensor:
        return torch.ones(shape, device=self.device) if "norm" in name else rnd(shape)

    def load_weights(self, tensors: dict[str, torch.Tensor]) -> None:
        self._load_globals(tensors)
        for gi, lw in enumerate(self.layers, self.start_layer):
            self._load_layer(lw, gi, tensors)

    @staticmethod
    def _take(tensors, name: str, shape: tuple) -> torch.Tensor:
        t = tensors.get(name)
        if t is None:
            raise KeyError(f"missing weight {name}")
        if t.dim() != len(shape) or any(s not in (-1, n) for s, n in zip(shape, t.shape)):
            raise ValueError(f"weight {name} has shape {tuple(t.shape)}, the config says {tuple(shape)}")
        return t

    def _getter(self, gi: int, tensors):
        """``get(name)``: checked tensor of layer ``gi`` on the stage's device."""
        shapes, p = self.weight_shapes(gi), f"l{gi}."

        def get(name, dtype=self.dtype):
            return self._take(tensors, p + name, shapes[p + name]).to(device=self.device, dtype=dtype).contiguous()

        return get

    def _global_getter(self, tensors):
        """``get(name)``: checked tensor outside the layers on the stage's device."""
        shapes = self.global_shapes()

        def get(name, dtype=self.dtype):
            return self._take(tensors, name, shapes[name]).to(device=self.device, dtype=dtype).contiguous()

        return get

    def _load_globals(self, tensors) -> None:
        get = self._global_getter(tensors)
        if self.is_first:
            self.embed = get("embed")
            if self.cfg.bigram is not None:
                self.bigram = get("bigram")
        if self.is_last:
            self.norm_w = get("final.norm", torch.float32)
            table = (self.embed if self.is_first else get("embed")) if self.cfg.tie_word_embeddings else get("head")
            self.lm_head = pad_rows(table, 8)

    def update_weights(self, tensors) -> int:
        """Online refit: layers named in ``tensors`` are rebuilt by the loader and moved into the live weights."""
        return self.reload_layers(tensors)

    def weight_bytes(self) -> int:
        ts = []
        shared = self.lm_head is not None and self.lm_head is self.embed
        for t in (getattr(self, name) for name in self._GLOBAL_TENSORS if not (shared and name == "lm_head")):
            ts += t.tensors() if hasattr(t, "tensors") else [] if t is None else [t]
        ts += [t for lw in self.layers for t in lw.tensors()]
        return sum(t.numel() * t.element_size() for t in ts)

    # ------------------------------------------------------------------ forward
    def embed_tokens(self, fb: ForwardBatch) -> torch.Tensor:
        b = self.cfg.bigram
        if b is None:
            return ops.embed_rows(self.embed, fb.input_ids, self.cfg.embedding_scale)
        return ops.embed_rows(self.embed, fb.input_ids, self.cfg.embedding_scale, self.bigram, fb.prev_ids,
                              b.mul_prev, b.mul_cur, b.buckets)

    def logits(self, h: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        rows = fb.logit_rows if fb.num_logits else None
        hn = ops.row_norm(h[:0] if rows is None else h, self.norm_w, self.cfg.rms_norm_eps, self.final_norm, rows=rows,
                          dtype=self.dtype, groups=self.cfg.norm_groups)
        return ops.linear(hn, self.lm_head, epi=ops.EPI_F32)[:, :self.cfg.vocab_size]
