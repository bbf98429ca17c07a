"""Pipeline-stage model for decoders that list their layers one by one and run some of them several times in a row
(``Zasalix``).

* A loop: layers ``start .. stop - 1`` run ``times`` times with the same weights, every pass with its own pages and state
  (:attr:`LayerCache.passes`). A later pass starts with the embedding added to the residual once more; every pass with a
  learned vector of its own.
* Sublayers are normed before and after, ``x += norm1b(mixer(norm1(x)))``, by tanh norms without statistics
  (:class:`TanhNorm`).
* Mixers: latent attention (:func:`latent_mix`), matrix memories (mLSTM, state per request), and both kinds side by side:
  windowed attention that keeps the first tokens in view, beside a matrix memory.
* Feed-forwards: dense (square of relu), or routed experts whose weights scale their input, with a shared expert.
* Behind the feed-forward a layer adds an input of its own for the token: a row of a side table, gated by the residual.

What is fused: the projections that read the same rows; rotation and the cache scatter; the memory's gates, scan and
normaliser into its kernel; norm, gate and factor of the heads; the output projections of two mixers side by side into ONE
product; activations into their products' epilogues; and everything that happens to the fp32 residual between two products
(:func:`ops.residual_step`: the sum of the experts' rows, the norm behind a sublayer, a pass's additions, the norm ahead of
the next one).
"""

from __future__ import annotations

from typing import Optional

import torch

from parallax_b200 import ops
from parallax_b200.engine.batch import ForwardBatch
from parallax_b200.models.latent import LATENT_SLOTS, latent_mix, latent_shapes, load_latent
from parallax_b200.models.layer_list import LayerListStage, ListedLayer, pad_rows
from parallax_b200.models.layer_spec import (ACT_GELU_TANH, MEMORY_SLICE, AttentionSpec, DenseSpec, LatentAttentionSpec,
                                             MatrixMemorySpec, ParallelSpec, RoutedSpec)
from parallax_b200.models.moe import RoutedExperts

_pad = torch.nn.functional.pad


def _up(n: int, multiple: int = 8) -> int:
    return n + -n % multiple


class TanhNorm:
    """``tanh(alpha x) w + b``."""

    __slots__ = ("w", "b", "alpha")

    def __init__(self, w, b, alpha):
        self.w, self.b, self.alpha = w, b, alpha

    @classmethod
    def load(cls, name: str, get) -> "TanhNorm":
        return cls(get(name, torch.float32), get(name + ".b", torch.float32), float(get(name + ".alpha", torch.float32)))

    @staticmethod
    def shapes(name: str, width: int) -> dict[str, tuple]:
        return {name: (width,), name + ".b": (width,), name + ".alpha": ()}

    def tensors(self) -> list:
        return [self.w, self.b]

    def args(self) -> tuple:
        return self.w, self.b, self.alpha


class LoopedLayer(ListedLayer):
    __slots__ = LATENT_SLOTS + ("norm1", "norm1b", "norm2", "norm2b", "offs", "w_gates", "b_gates", "mem_norm", "w_up", "w_gu",
                                "w_down", "moe", "side_gate", "side_proj", "side_norm")


class LoopedStage(LayerListStage):
    layer_class = LoopedLayer
    _GLOBAL_KEYS = LayerListStage._GLOBAL_KEYS + ("final.norm.b", "final.norm.alpha", "side.embed", "loop.step")
    _GLOBAL_TENSORS = ("embed", "final", "lm_head", "side_table", "loop_step")
    _TABLES_EVERYWHERE = True

    def __init__(self, cfg, start_layer: int, end_layer: int, *args, **kwargs):
        loop = cfg.loop
        if loop is not None and loop.times > 1 and 0 < start_layer < loop.stop:
            raise ValueError(f"layers 0 to {loop.stop - 1} must be in one pipeline stage (later passes of the loop start from the "
                             f"embedding again), but one starts with layer {start_layer}")
        if loop is not None and loop.times > 1 and start_layer == 0 and end_layer < loop.stop:
            raise ValueError(f"layers 0 to {loop.stop - 1} must be in one pipeline stage, this one ends with layer {end_layer - 1}")
        super().__init__(cfg, start_layer, end_layer, *args, **kwargs)
        self.final: Optional[TanhNorm] = None
        self.side_table: Optional[torch.Tensor] = None    # [vocab, layers of the stage * side_cols]
        self.loop_step: Optional[torch.Tensor] = None     # [passes, width] fp32
        self.side_cols = _up(cfg.token_side_dim)
        self._span = (start_layer, end_layer)
        self._layers_only = False
        # (local layer, pass) in the order they run
        span = range(start_layer, end_layer)
        inside = [gi for gi in span if loop is not None and loop.start <= gi < loop.stop]
        before, after = [gi for gi in span if inside and gi < inside[0]], [gi for gi in span if not inside or gi > inside[-1]]
        passes = [(gi, t) for t in range(loop.times if inside else 0) for gi in inside]
        self.runs = [(gi - start_layer, t) for gi, t in [(g, 0) for g in before] + passes + [(g, 0) for g in after]]

    def attach_kv(self, kv_caches: list) -> None:
        if any(lc.k is not None and lc.k.dtype != self.dtype for lc in kv_caches):
            raise ValueError(f"{self.cfg.architecture} keeps its keys and values in {self.dtype} (no quantised pages)")
        super().attach_kv(kv_caches)

    # ------------------------------------------------------------------ weights
    def global_shapes(self) -> dict[str, tuple]:
        cfg, sh = self.cfg, super().global_shapes()
        if self.is_last:
            sh.update(TanhNorm.shapes("final.norm", cfg.hidden_size))
        if cfg.token_side_dim:
            sh["side.embed"] = (cfg.vocab_size, cfg.num_hidden_layers * cfg.token_side_dim)
        if cfg.loop is not None:
            sh["loop.step"] = (cfg.loop.times, cfg.hidden_size)
        return sh

    def _prepare_shadow(self, shadow) -> None:
        shadow._layers_only = bool(shadow.layers)      # a stage that reloads one layer leaves the tables alone

    def _load_globals(self, tensors) -> None:
        if self._layers_only:
            return
        cfg, get = self.cfg, self._global_getter(tensors)
        if self.is_first:
            self.embed = get("embed")
        if self.is_last:
            self.final, self.lm_head = TanhNorm.load("final.norm", get), pad_rows(get("head"), 8)
        if cfg.token_side_dim:
            d, (lo, hi) = cfg.token_side_dim, self._span
            rows = get("side.embed").view(cfg.vocab_size, cfg.num_hidden_layers, d)[:, lo:hi]
            self.side_table = _pad(rows, (0, self.side_cols - d)).reshape(cfg.vocab_size, -1).contiguous()
        if cfg.loop is not None:
            self.loop_step = get("loop.step", torch.float32)

    @staticmethod
    def _memory_shapes(m: MatrixMemorySpec, W: int) -> dict[str, tuple]:
        sh = {"q": (m.q_rows, W), "k": (m.k_rows, W), "v": (m.v_rows, W), "g": (m.out_width, W), "o": (W, m.out_width),
              "norm": (m.out_width,)}
        for n in "if":
            sh.update({n: (m.heads, W), n + ".b": (m.heads,)})
        return sh

    @staticmethod
    def _attention_shapes(m: AttentionSpec, W: int) -> dict[str, tuple]:
        return {"q": (m.q_rows, W), "k": (m.k_rows, W), "v": (m.v_rows, W), "g": (m.out_width, W), "o": (W, m.out_width)}

    def weight_shapes(self, gi: int) -> dict[str, tuple]:
        W, spec, p = self.cfg.hidden_size, self.cfg.layer_specs[gi], f"l{gi}."
        m, mlp, sh = spec.mixer, spec.mlp, {}
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp is not None else ()):
            sh.update(TanhNorm.shapes(p + n, W))
        if isinstance(m, LatentAttentionSpec):
            mix = latent_shapes(m, W)
        elif isinstance(m, MatrixMemorySpec):
            mix = self._memory_shapes(m, W)
        else:
            mix = {"left." + n: s for n, s in self._attention_shapes(m.left, W).items()}
            mix.update({"right." + n: s for n, s in self._memory_shapes(m.right, W).items()})
        sh.update({p + "mix." + n: s for n, s in mix.items()})
        if self.cfg.token_side_dim:
            d = self.cfg.token_side_dim
            sh.update({p + "side.gate": (d, W), p + "side.proj": (W, d), p + "side.norm": (W,)})

        def ffn(q, ff):
            sh.update({q + "gate": (ff, W), q + "up": (ff, W), q + "down": (W, ff)})

        if isinstance(mlp, DenseSpec):
            sh.update({p + "mlp.up": (mlp.ff, W), p + "mlp.down": (W, mlp.ff)})
        elif mlp is not None:
            sh[p + "mlp.router"] = (mlp.outputs, W)
            for e in range(mlp.experts):
                ffn(p + f"mlp.e{e}.", mlp.expert.ff)
            if mlp.shared:
                ffn(p + "mlp.shared.", mlp.shared.ff)
        return sh

    def _random(self, name: str, shape: tuple, rnd) -> torch.Tensor:
        if name.endswith(".alpha"):
            return torch.full(shape, 0.5, device=self.device)
        return torch.zeros(shape, device=self.device) if name.endswith(".b") else super()._random(name, shape, rnd)

    def _load_layer(self, lw: LoopedLayer, gi: int, tensors) -> None:
        self._describe(lw, gi)
        spec, get = lw.spec, self._getter(gi, tensors)
        m, mlp, cat, f32 = spec.mixer, spec.mlp, torch.cat, torch.float32
        lw.norm1, lw.norm1b = TanhNorm.load("norm1", get), TanhNorm.load("norm1b", get)
        if mlp is not None:
            lw.norm2, lw.norm2b = TanhNorm.load("norm2", get), TanhNorm.load("norm2b", get)
        if isinstance(m, LatentAttentionSpec):
            load_latent(lw, m, lambda n, dt=self.dtype: get("mix." + n, dt))
        else:
            left = "left." if isinstance(m, ParallelSpec) else None
            right = "right." if left else ""
            # the products that read h, one matrix, and where its parts start; every part on a multiple of 8 rows
            lw.offs, parts, at = {}, [], 0
            for n in ([left + n for n in "qkvg"] if left else []) + [right + n for n in "qkvg"]:
                parts.append(pad_rows(get("mix." + n), 8))
                lw.offs[n], at = at, at + parts[-1].shape[0]
            lw.w_in = cat(parts, 0).contiguous()
            # gates of the recurrence: a product of their own, whose result stays fp32
            lw.w_gates = pad_rows(cat([get(f"mix.{right}{n}") for n in "if"], 0), 8)
            lw.b_gates = cat([get(f"mix.{right}{n}.b", f32) for n in "if"], 0)
            lw.mem_norm = get(f"mix.{right}norm", f32)
            outs = [get("mix." + p + "o") for p in ((left, right) if left else (right,))]
            lw.w_o = cat([_pad(o, (0, -o.shape[1] % 8)) for o in outs], 1).contiguous()
        lw.moe = None
        if isinstance(mlp, DenseSpec):
            lw.w_up = pad_rows(get("mlp.up"), 8)
            lw.w_down = _pad(get("mlp.down"), (0, -mlp.ff % 8)).contiguous()
        elif mlp is not None:
            lw.moe = RoutedExperts.build(mlp, lambda n, dt=self.dtype: get("mlp." + n, dt), self.device)
            if mlp.shared:
                lw.w_gu = ops.interleave_gate_up(pad_rows(get("mlp.shared.gate"), 64), pad_rows(get("mlp.shared.up"), 64))
                lw.w_down = _pad(get("mlp.shared.down"), (0, -mlp.shared.ff % 64)).contiguous()
        if self.cfg.token_side_dim:
            lw.side_gate = pad_rows(get("side.gate"), 8)
            lw.side_proj = _pad(get("side.proj"), (0, -self.cfg.token_side_dim % 8)).contiguous()
            lw.side_norm = get("side.norm", f32)

    # ------------------------------------------------------------------ mixers
    def _attention(self, lw: LoopedLayer, m: AttentionSpec, offs: tuple, cache, proj, fb: ForwardBatch) -> torch.Tensor:
        """Heads ``[T, heads, columns]`` of the windowed attention; the first ``vdim`` columns count."""
        T = proj.shape[0]
        q = torch.empty((T, m.heads, m.head_cols), dtype=proj.dtype, device=proj.device)
        ops.conv_qkv_prep(proj, offs, m.heads, m.kv_heads, m.dim, m.vdim, None, None, None, None, lw.cos_sin, fb.positions,
                          fb.seq_cu, fb.seq_slots, fb.num_prefill_seqs, fb.num_prefill_tokens, fb.slot_mapping, cache.k, cache.v,
                          q, 0.0)
        heads, Tp = torch.empty_like(q), fb.num_prefill_tokens
        if Tp:
            ops.attn_prefill(q[:Tp], cache.k, cache.v, fb.p_block_tables, fb.p_cu_q, fb.p_ctx_lens, fb.p_max_q, m.scale,
                             window=m.window, keep_first=m.keep_first, out=heads[:Tp])
        if fb.num_decode:
            ops.attn_decode(q[Tp:], cache.k, cache.v, fb.d_block_tables, fb.d_ctx_lens, m.scale, window=m.window,
                            max_ctx=fb.d_max_ctx, keep_first=m.keep_first, out=heads[Tp:])
        return heads

    def _mixer(self, lw: LoopedLayer, cache, h: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        m, eps = lw.spec.mixer, self.cfg.rms_norm_eps
        if isinstance(m, LatentAttentionSpec):
            return latent_mix(lw, m, cache.k, h, fb, eps)
        both = isinstance(m, ParallelSpec)
        mem, right, scale = (m.right, "right.", m.right_scale) if both else (m, "", 1.0)
        o, proj, gates = lw.offs, ops.linear(h, lw.w_in), ops.linear(h, lw.w_gates, epi=ops.EPI_F32)
        cat, at = torch.empty((h.shape[0], lw.w_o.shape[1]), dtype=h.dtype, device=h.device), 0
        if both:
            a = m.left
            heads = self._attention(lw, a, (o["left.q"], o["left.k"], o["left.v"]), cache, proj, fb)
            at = _up(a.out_width)
            ops.gated_rows(heads, a.vdim, proj[:, o["left.g"]:o["left.g"] + a.out_width], cat[:, :at], scale=m.left_scale)
        heads = ops.matrix_memory(proj, (o[right + "q"], o[right + "k"], o[right + "v"]), mem.heads, mem.dim, mem.vdim, gates,
                                  lw.b_gates, mem.gate_cap, cache.rec_state, fb.positions, fb.seq_cu, fb.seq_slots,
                                  fb.num_prefill_seqs, MEMORY_SLICE)
        ops.gated_rows(heads, mem.vdim, proj[:, o[right + "g"]:o[right + "g"] + mem.out_width], cat[:, at:], lw.mem_norm, eps,
                       per_head=True, scale=scale)
        return ops.linear(cat, lw.w_o)

    # ------------------------------------------------------------------ forward
    def _feed_forward(self, lw: LoopedLayer, h: torch.Tensor):
        """(rows of the dense or shared feed-forward or None, expert rows or None)."""
        mlp = lw.spec.mlp
        if isinstance(mlp, DenseSpec):
            return ops.linear(ops.act_linear(h, lw.w_up, mlp.act), lw.w_down), None
        routed, _ = lw.moe.forward(h)
        return (ops.linear(ops.glu_linear(h, lw.w_gu, mlp.shared.act), lw.w_down) if mlp.shared else None), routed

    def _entry(self, run: int, fb: ForwardBatch) -> dict:
        """What is added to the residual ahead of run number ``run``."""
        if run >= len(self.runs):
            return {}
        li, t = self.runs[run]
        loop = self.cfg.loop
        if loop is None or li + self.start_layer != loop.start:
            return {}
        again = dict(table=self.embed, ids=fb.input_ids) if t else {}
        return dict(step=self.loop_step[t], **again)

    def forward_layers(self, x: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        eps, dt, side = self.cfg.rms_norm_eps, self.dtype, self.cfg.token_side_dim
        if not self.is_first:
            x = x.clone()       # the residual is updated in place; the incoming buffer belongs to the caller
        h = ops.residual_step(x, pre=self.layers[self.runs[0][0]].norm1.args(), dtype=dt, **self._entry(0, fb))
        for r, (li, t) in enumerate(self.runs):
            lw = self.layers[li]
            y, routed, post = self._mixer(lw, self.kv_caches[li].passes[t], h, fb), None, lw.norm1b
            if lw.spec.mlp is not None:
                h = ops.residual_step(x, y, post.args(), pre=lw.norm2.args(), dtype=dt)
                (y, routed), post = self._feed_forward(lw, h), lw.norm2b
            leave = dict(pre=self.layers[self.runs[r + 1][0]].norm1.args() if r + 1 < len(self.runs) else None, dtype=dt,
                         **self._entry(r + 1, fb))
            if not side:
                h = ops.residual_step(x, y, post.args(), routed, **leave)
                continue
            low = ops.residual_step(x, y, post.args(), routed, pre=(), dtype=dt)
            g = ops.act_linear(low, lw.side_gate, ACT_GELU_TANH, self.side_table, fb.input_ids, li * self.side_cols)
            h = ops.residual_step(x, ops.linear(g, lw.side_proj), (lw.side_norm,), eps=eps, **leave)
        return x

    def logits(self, h: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        hn = ops.tanh_norm(h, *self.final.args(), rows=fb.logit_rows, dtype=self.dtype)
        return ops.linear(hn, self.lm_head, epi=ops.EPI_F32)[:, :self.cfg.vocab_size]
