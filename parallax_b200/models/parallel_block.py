"""Pipeline-stage model for decoders that list their layers one by one and run each layer's token mixer and
feed-forward side by side (``Zudepel``): with ``h = rmsnorm(x)``, ``x += mixer(h) + feed_forward(h)``.

* Mixers: softmax attention (short convolutions on q, k and v, norms over the whole q and k rows, half-split
  rotation, sinks, output gate; a layer may read an earlier layer's cached keys and values) and lightning attention
  (linear attention with a fixed decay per head, state per request).
* Feed-forwards: dense gated (GELU), or routed experts (identity experts, groups, correction) with a gated shared
  expert; a layer may have none.

What is fused: the projections that read ``h`` (queries | keys | values | gate); convolution, norms, rotation and the
cache scatter (:func:`ops.conv_qkv_prep`); the gated activation into its product's epilogue, with the shared expert's
gate; the output projection and the (dense or shared) down projection into ONE product, whose operand columns are the
gated heads and the activations; the residual update, the weighted sum of the experts' rows and the next layer's norm
(:func:`ops.residual_add`). The residual is fp32 (``hidden_dtype``).
"""

from __future__ import annotations

from typing import Optional

import torch

from parallax_b200 import ops
from parallax_b200.engine.batch import ForwardBatch
from parallax_b200.models.layer_list import LayerListStage, ListedLayer, pad_rows
from parallax_b200.models.layer_spec import AttentionSpec, GLUSpec, RoutedSpec
from parallax_b200.models.moe import RoutedExperts

_CHUNK = 64      # tokens of one step of the chunked lightning kernel: powers of the decay up to this are tabulated


def _up(n: int, multiple: int) -> int:
    return n + -n % multiple


class ParallelLayer(ListedLayer):
    __slots__ = ("norm1", "w_in", "b_in", "offs", "conv_w", "q_norm", "k_norm", "sinks", "decay_pow", "mix_norm", "w_gu",
                 "w_out", "moe")


class ParallelBlockStage(LayerListStage):
    layer_class = ParallelLayer
    final_norm = ops.NORM_RMS

    def __init__(self, cfg, start_layer: int, end_layer: int, *args, **kwargs):
        for gi in range(start_layer, end_layer):
            src = cfg.layer_specs[gi].mixer.kv_from
            if src is not None and src < start_layer:
                raise ValueError(f"layer {gi} reads the keys of layer {src}: both must be in one pipeline stage, this one "
                                 f"has layers {start_layer} to {end_layer - 1}")
        super().__init__(cfg, start_layer, end_layer, *args, **kwargs)

    def attach_kv(self, kv_caches: list) -> None:
        if any(lc.k is not None and lc.k.dtype != self.dtype for lc in kv_caches):
            raise ValueError(f"{self.cfg.architecture} keeps its keys and values in {self.dtype} (no quantised pages)")
        super().attach_kv(kv_caches)

    # ------------------------------------------------------------------ weights
    @staticmethod
    def _parts(m) -> dict[str, int]:
        """Rows of the packed input projection, part by part."""
        parts = {"q": m.q_rows, "k": m.k_rows, "v": m.v_rows, "g": m.out_width}
        return {n: r for n, r in parts.items() if r}

    @staticmethod
    def _tail(mlp) -> Optional[GLUSpec]:
        """The feed-forward that every token runs: dense, or the shared expert."""
        return mlp.shared if isinstance(mlp, RoutedSpec) else mlp

    def weight_shapes(self, gi: int) -> dict[str, tuple]:
        W, spec = self.cfg.hidden_size, self.cfg.layer_specs[gi]
        m, p = spec.mixer, f"l{gi}."
        sh = {p + "norm1": (W,), p + "mix.o": (W, m.out_width)}
        for name, rows in self._parts(m).items():
            sh[p + "mix." + name] = (rows, W)
            if isinstance(m, AttentionSpec) and name != "g":
                sh[p + f"mix.{name}.b"] = (rows,)
                if m.conv:
                    sh[p + f"mix.{name}.conv"] = (rows, m.conv)
                if name != "v":
                    sh[p + f"mix.{name}.norm"] = (rows,)
        if isinstance(m, AttentionSpec):
            sh[p + "mix.sink"] = (m.heads,)
        else:
            sh[p + "mix.norm"] = (m.out_width,)

        def ffn(q, ff):
            sh.update({q + "gate": (ff, W), q + "up": (ff, W), q + "down": (W, ff)})

        if isinstance(spec.mlp, RoutedSpec):
            r = spec.mlp
            sh.update({p + "mlp.router": (r.outputs, W), p + "mlp.correction": (r.outputs,)})
            for e in range(r.experts):
                ffn(p + f"mlp.e{e}.", r.expert.ff)
            if r.shared:
                ffn(p + "mlp.shared.", r.shared.ff)
                sh[p + "mlp.shared.sg"] = (1, W)
        elif spec.mlp is not None:
            ffn(p + "mlp.", spec.mlp.ff)
        return sh

    def _load_layer(self, lw: ParallelLayer, gi: int, tensors) -> None:
        self._describe(lw, gi)
        spec, get = lw.spec, self._getter(gi, tensors)
        m, cat = spec.mixer, torch.cat
        parts = self._parts(m)
        lw.norm1 = get("norm1", torch.float32)
        # the products that read h, one matrix; every part starts on a multiple of 8 rows
        lw.w_in = cat([pad_rows(get("mix." + n), 8) for n in parts], 0).contiguous()
        offs, o = {}, 0
        for n, rows in parts.items():
            offs[n], o = o, o + _up(rows, 8)
        lw.offs = offs
        if isinstance(m, AttentionSpec):
            lw.b_in = cat([pad_rows(get(f"mix.{n}.b") if n != "g" else lw.w_in.new_zeros(r), 8) for n, r in parts.items()])
            convolved = [n for n in parts if n != "g"]
            lw.conv_w = cat([get(f"mix.{n}.conv") for n in convolved], 0).t().contiguous() if m.conv else None
            lw.q_norm = get("mix.q.norm", torch.float32)
            lw.k_norm = get("mix.k.norm", torch.float32) if "k" in parts else None
            lw.sinks = get("mix.sink", torch.float32)
        else:
            n = torch.arange(_CHUNK + 1, dtype=torch.float64)
            lw.decay_pow = (torch.tensor(m.decay, dtype=torch.float64)[:, None] ** n).float().to(self.device).contiguous()
            lw.mix_norm = get("mix.norm", torch.float32)
        # output projection and the down projection of the feed-forward every token runs, side by side: columns
        # [heads, padded to 8 | activations, padded to 64]
        pad = torch.nn.functional.pad
        outs = [pad(get("mix.o"), (0, -m.out_width % 8))]
        tail = self._tail(spec.mlp)
        if tail is not None:
            t = "mlp.shared." if isinstance(spec.mlp, RoutedSpec) else "mlp."
            lw.w_gu = ops.interleave_gate_up(pad_rows(get(t + "gate"), 64), pad_rows(get(t + "up"), 64))
            outs.append(pad(get(t + "down"), (0, -tail.ff % 64)))
        lw.w_out = cat(outs, 1).contiguous()
        lw.moe = None
        if isinstance(spec.mlp, RoutedSpec):
            lw.moe = RoutedExperts.build(spec.mlp, lambda n, dt=self.dtype: get("mlp." + n, dt), self.device)

    # ------------------------------------------------------------------ forward
    def _attention(self, lw: ParallelLayer, li: int, h: torch.Tensor, fb: ForwardBatch, out: torch.Tensor) -> None:
        m, T, offs = lw.spec.mixer, h.shape[0], lw.offs
        own = self.kv_caches[li]
        src = own if m.kv_from is None else self.kv_caches[m.kv_from - self.start_layer]
        proj = ops.linear(h, lw.w_in, bias=lw.b_in)
        q = torch.empty((T, m.heads, m.head_cols), dtype=h.dtype, device=h.device)
        ops.conv_qkv_prep(proj, (offs["q"], offs.get("k", 0), offs.get("v", 0)), m.heads, m.kv_heads, m.dim, m.vdim, lw.conv_w,
                          own.conv_state, lw.q_norm, lw.k_norm, lw.cos_sin, fb.positions, fb.seq_cu, fb.seq_slots,
                          fb.num_prefill_seqs, fb.num_prefill_tokens, fb.slot_mapping, own.k, own.v, q,
                          self.cfg.rms_norm_eps)
        heads = torch.empty_like(q)
        Tp = fb.num_prefill_tokens
        if Tp:
            ops.attn_prefill(q[:Tp], src.k, src.v, fb.p_block_tables, fb.p_cu_q, fb.p_ctx_lens, fb.p_max_q, m.scale,
                             sinks=lw.sinks, out=heads[:Tp])
        if fb.num_decode:
            ops.attn_decode(q[Tp:], src.k, src.v, fb.d_block_tables, fb.d_ctx_lens, m.scale, sinks=lw.sinks,
                            max_ctx=fb.d_max_ctx, out=heads[Tp:])
        ops.gated_rows(heads, m.vdim, proj[:, offs["g"]:offs["g"] + m.out_width], out)

    def _lightning(self, lw: ParallelLayer, li: int, h: torch.Tensor, fb: ForwardBatch, out: torch.Tensor) -> None:
        m, offs = lw.spec.mixer, lw.offs
        proj = ops.linear(h, lw.w_in)
        heads = ops.lightning_attn(proj, (offs["q"], offs["k"], offs["v"]), m.heads, m.dim, m.vdim, lw.decay_pow,
                                   self.kv_caches[li].rec_state, fb.positions, fb.seq_cu, fb.seq_slots, fb.num_prefill_seqs)
        ops.gated_rows(heads, m.vdim, proj[:, offs["g"]:offs["g"] + m.out_width], out, lw.mix_norm, self.cfg.rms_norm_eps)

    def forward_layers(self, x: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        eps = self.cfg.rms_norm_eps
        if not self.is_first:
            x = x.clone()       # the residual is updated in place; the incoming buffer belongs to the caller
        h = ops.row_norm(x, self.layers[0].norm1, eps, ops.NORM_RMS, dtype=self.dtype)
        for li, lw in enumerate(self.layers):
            m = lw.spec.mixer
            heads_cols = _up(m.out_width, 8)
            cat = torch.empty((x.shape[0], lw.w_out.shape[1]), dtype=h.dtype, device=h.device)
            mix = self._attention if isinstance(m, AttentionSpec) else self._lightning
            mix(lw, li, h, fb, cat[:, :heads_cols])
            routed = gate = None
            if lw.moe is not None:
                routed, gate = lw.moe.forward(h)
            tail = self._tail(lw.spec.mlp)
            if tail is not None:
                ops.glu_linear(h, lw.w_gu, tail.act, gate, cat[:, heads_cols:])
            y = ops.linear(cat, lw.w_out)
            nxt = self.layers[li + 1].norm1 if li + 1 < len(self.layers) else None
            h = ops.residual_add(x, y, nxt, eps, routed, h)
        return x
