"""Pipeline-stage model for pre-norm decoders that list their layers one by one and mix three kinds of token mixers
(``Kikurax``): ``x += mixer(norm1(x))``, ``x += feed_forward(norm2(x))``, RMS norms over equal parts of the row.

* Softmax attention: rotation with stretched frequencies, q and k over their root mean square per head, a temperature per
  head, soft-capped scores, one added to the denominator; a layer's values are mixed with those of the first such layer.
* State-space layers (Mamba-2): short convolution, scalar decay per head, gate ahead of a grouped norm.
* Two mixers side by side: attention whose weights are sigmoids (no rotation; queries grow with the logarithm of the position),
  with an output gate, and a gated delta rule with a decay per key channel behind short convolutions. Their outputs are normed
  over the model width and averaged.
* Feed-forward: routed experts with clipped gated activations, chosen by biased logits. The output head is the embedding table.

What is fused: the projections that read the same rows; rotation, norms, temperatures, value mixing and the cache scatter
(:func:`ops.head_qkv_prep`); convolution, bias and SiLU; decays, step sizes, unit norms and the recurrences; gate and norm of the
heads; activations into their products' epilogues; and the residual update (one output, two normed outputs, or the weighted
expert rows) with the next norm (:func:`ops.residual_add`). The residual is fp32 (``hidden_dtype``).
"""

from __future__ import annotations

import torch

from parallax_b200 import ops
from parallax_b200.engine.batch import ForwardBatch
from parallax_b200.models.layer_list import LayerListStage, ListedLayer, pad_rows
from parallax_b200.models.layer_spec import AttentionSpec, DeltaSpec, ParallelSpec, StateSpaceSpec
from parallax_b200.models.moe import RoutedExperts

_pad = torch.nn.functional.pad


def _pack(parts: dict) -> tuple:
    """(one matrix of the parts' rows, where each starts); every part on a multiple of 8 rows."""
    offs, rows, at = {}, [], 0
    for n, w in parts.items():
        rows.append(pad_rows(w, 8))
        offs[n], at = at, at + rows[-1].shape[0]
    return torch.cat(rows, 0).contiguous(), offs


def _pad_columns(w: torch.Tensor, multiple: int = 8) -> torch.Tensor:
    return _pad(w, (0, -w.shape[1] % multiple)).contiguous()


class PreNormLayer(ListedLayer):
    __slots__ = ("norm1", "norm2", "w_in", "b_in", "offs", "w_o", "moe",
                 # attention: factor of every query head, share of the first layer's values, bias of sigmoid weights, factor of
                 # the queries at every position
                 "head_scale", "v_mix", "sinks", "sig_bias", "pos_scale",
                 # recurrences: taps [taps, channels] and their bias, logits that stay fp32, decay and step parameters
                 "conv_w", "conv_b", "w_step", "dt_bias", "A_log", "D", "head_norm", "w_decay", "w_gate",
                 # two mixers: output projection of the second, norms of both outputs
                 "w_o2", "norm_left", "norm_right")


class PreNormStage(LayerListStage):
    layer_class = PreNormLayer
    final_norm = ops.NORM_RMS

    def __init__(self, cfg, start_layer: int, end_layer: int, *args, **kwargs):
        for gi in range(start_layer, end_layer):
            src = getattr(cfg.layer_specs[gi].mixer, "v_first", None)
            if src is not None and src < start_layer:
                raise ValueError(f"layer {gi} mixes in the values of layer {src}: both must be in one pipeline stage, this one "
                                 f"has layers {start_layer} to {end_layer - 1}")
        super().__init__(cfg, start_layer, end_layer, *args, **kwargs)

    def attach_kv(self, kv_caches: list) -> None:
        if any(lc.k is not None and lc.k.dtype != self.dtype for lc in kv_caches):
            raise ValueError(f"{self.cfg.architecture} keeps its keys and values in {self.dtype} (no quantised pages)")
        super().attach_kv(kv_caches)

    # ------------------------------------------------------------------ weights
    @staticmethod
    def _attention_shapes(m: AttentionSpec, W: int) -> dict[str, tuple]:
        return {"q": (m.q_rows, W), "k": (m.k_rows, W), "v": (m.v_rows, W), "o": (W, m.out_width)}

    @staticmethod
    def _delta_shapes(m: DeltaSpec, W: int) -> dict[str, tuple]:
        sh = {"o": (W, m.out_width), "b": (m.heads, W), "A_log": (m.heads,), "dt_bias": (m.heads * m.dim,), "norm": (m.vdim,),
              "a1": (-1, W), "a2": (m.heads * m.dim, -1), "g1": (-1, W), "g2": (m.out_width, -1)}
        for n, rows in (("q", m.q_rows), ("k", m.k_rows), ("v", m.v_rows)):
            sh.update({n: (rows, W), n + ".conv": (rows, m.conv)})
        return sh

    @staticmethod
    def _state_space_shapes(m: StateSpaceSpec, W: int) -> dict[str, tuple]:
        convolved = m.out_width + 2 * m.bc_rows
        return {"in": (m.out_width + convolved + m.heads, W), "conv": (convolved, m.conv), "conv.b": (convolved,),
                "dt_bias": (m.heads,), "A_log": (m.heads,), "D": (m.heads,), "norm": (m.out_width,), "o": (W, m.out_width)}

    def weight_shapes(self, gi: int) -> dict[str, tuple]:
        W, spec, p = self.cfg.hidden_size, self.cfg.layer_specs[gi], f"l{gi}."
        m, mlp = spec.mixer, spec.mlp
        if isinstance(m, ParallelSpec):
            left = dict(self._attention_shapes(m.left, W), g=(m.left.out_width, W), pb=(m.left.heads,), out=(W,))
            right = dict(self._delta_shapes(m.right, W), out=(W,))
            mix = {**{"left." + n: s for n, s in left.items()}, **{"right." + n: s for n, s in right.items()}}
        elif isinstance(m, StateSpaceSpec):
            mix = self._state_space_shapes(m, W)
        else:
            mix = dict(self._attention_shapes(m, W), temp=(m.heads,), **{"q.b": (m.q_rows,), "k.b": (m.k_rows,), "v.b": (m.v_rows,)})
            if m.v_first is not None:
                mix["vmix"] = ()
        sh = {p + "norm1": (W,), **{p + "mix." + n: s for n, s in mix.items()}}
        if mlp is not None:
            sh.update({p + "norm2": (W,), p + "mlp.router": (mlp.outputs, W), p + "mlp.router.b": (mlp.outputs,)})
            for e in range(mlp.experts):
                q = p + f"mlp.e{e}."
                sh.update({q + "gate": (mlp.ff, W), q + "up": (mlp.ff, W), q + "down": (W, mlp.ff)})
        return sh

    def _random(self, name: str, shape: tuple, rnd) -> torch.Tensor:
        if name.endswith((".out", ".temp", ".D")):
            return torch.ones(shape, device=self.device)
        if name.endswith(".vmix"):
            return torch.full(shape, 0.5, device=self.device)
        return super()._random(name, tuple(max(8, self.cfg.hidden_size // 32) if n < 0 else n for n in shape), rnd)

    def _load_attention(self, lw: PreNormLayer, m: AttentionSpec, get) -> None:
        lw.w_in, lw.offs = _pack({n: get(n) for n in "qkv"})
        lw.b_in = torch.cat([pad_rows(get(n + ".b"), 8) for n in "qkv"])
        lw.head_scale = get("temp", torch.float32)
        lw.v_mix = float(get("vmix", torch.float32)) if m.v_first is not None else 0.0
        lw.sinks = torch.zeros(m.heads, dtype=torch.float32, device=self.device)    # a score of 0 without a value
        # columns for the padding of the heads: the product reads them as the attention leaves them
        o = get("o").view(-1, m.heads, m.vdim)
        lw.w_o = _pad(o, (0, m.head_cols - m.vdim)).reshape(o.shape[0], -1).contiguous()

    def _load_state_space(self, lw: PreNormLayer, m: StateSpaceSpec, get) -> None:
        sizes = [m.out_width, m.out_width, m.bc_rows, m.bc_rows, m.heads]
        z, x, b, c, dt = get("in").split(sizes, 0)
        lw.w_in, lw.offs = _pack({"z": z, "x": x, "B": b, "C": c})
        lw.w_step = pad_rows(dt, 8)
        lw.conv_w = torch.cat([pad_rows(t, 8) for t in get("conv").split(sizes[1:4], 0)], 0).t().contiguous()
        lw.conv_b = torch.cat([pad_rows(t, 8) for t in get("conv.b").split(sizes[1:4], 0)])
        lw.dt_bias, lw.A_log, lw.D, lw.head_norm = (get(n, torch.float32) for n in ("dt_bias", "A_log", "D", "norm"))
        lw.w_o = _pad_columns(get("o"))

    def _load_parallel(self, lw: PreNormLayer, m: ParallelSpec, get) -> None:
        a, f32 = m.left, torch.float32
        for n in ("a", "g"):
            if get(f"right.{n}1").shape[0] != get(f"right.{n}2").shape[1]:
                raise ValueError(f"layer {lw.layer_idx}: mix.right.{n}1 and mix.right.{n}2 do not fit together")
        names = ["left." + n for n in "qkvg"] + ["right." + n for n in ("q", "k", "v", "a1", "g1")]
        lw.w_in, lw.offs = _pack({n: get(n) for n in names})
        lw.sig_bias = get("left.pb", f32)
        if a.q_temp is not None:
            coef, every = a.q_temp
            p = torch.arange(1, self.max_positions + 1, dtype=torch.float64)
            lw.pos_scale = (1 + coef * torch.log(torch.floor(p / every) + 1)).float().to(self.device)
        lw.conv_w = torch.cat([pad_rows(get(f"right.{n}.conv"), 8) for n in "qkv"], 0).t().contiguous()
        lw.w_step = pad_rows(get("right.b"), 8)
        lw.w_decay, lw.w_gate = (_pad_columns(pad_rows(get("right." + n), 8)) for n in ("a2", "g2"))
        lw.dt_bias, lw.A_log = get("right.dt_bias", f32), get("right.A_log", f32)
        lw.head_norm = get("right.norm", f32).repeat(m.right.heads).contiguous()
        lw.w_o, lw.w_o2 = _pad_columns(get("left.o")), _pad_columns(get("right.o"))
        lw.norm_left, lw.norm_right = get("left.out", f32), get("right.out", f32)

    def _load_layer(self, lw: PreNormLayer, gi: int, tensors) -> None:
        self._describe(lw, gi)
        get, m, mlp = self._getter(gi, tensors), lw.spec.mixer, lw.spec.mlp
        load = self._load_parallel if isinstance(m, ParallelSpec) else \
            self._load_state_space if isinstance(m, StateSpaceSpec) else self._load_attention
        load(lw, m, lambda n, dt=self.dtype: get("mix." + n, dt))
        lw.norm1, lw.norm2, lw.moe = get("norm1", torch.float32), None, None
        if mlp is not None:
            lw.norm2 = get("norm2", torch.float32)
            lw.moe = RoutedExperts.build(mlp, lambda n, dt=self.dtype: get("mlp." + n, dt), self.device)

    # ------------------------------------------------------------------ mixers
    def _attend(self, lw: PreNormLayer, m: AttentionSpec, offs: tuple, cache, proj, fb: ForwardBatch, v_first=None) -> torch.Tensor:
        """Heads ``[T, heads, columns]``; the first ``vdim`` columns count, zeros behind."""
        q = torch.empty((proj.shape[0], m.heads, m.head_cols), dtype=proj.dtype, device=proj.device)
        ops.head_qkv_prep(proj, offs, m.heads, m.kv_heads, m.dim, m.vdim, self.cfg.rms_norm_eps, lw.cos_sin, fb.positions,
                          fb.slot_mapping, cache.k, cache.v, q, lw.head_scale, lw.pos_scale, v_first, lw.v_mix or 0.0)
        heads, Tp = torch.empty_like(q), fb.num_prefill_tokens
        score = dict(sinks=lw.sinks, softcap=m.softcap, sigmoid_bias=lw.sig_bias)
        if Tp:
            ops.attn_prefill(q[:Tp], cache.k, cache.v, fb.p_block_tables, fb.p_cu_q, fb.p_ctx_lens, fb.p_max_q, m.scale,
                             out=heads[:Tp], **score)
        if fb.num_decode:
            ops.attn_decode(q[Tp:], cache.k, cache.v, fb.d_block_tables, fb.d_ctx_lens, m.scale, max_ctx=fb.d_max_ctx,
                            out=heads[Tp:], **score)
        return heads

    def _convolve(self, lw: PreNormLayer, cache, x, fb: ForwardBatch) -> torch.Tensor:
        return ops.short_conv(x, lw.conv_w, lw.conv_b, cache.conv_state, fb.positions, fb.seq_cu, fb.seq_slots, fb.num_prefill_seqs,
                              fb.num_prefill_tokens)

    def _state_space(self, lw: PreNormLayer, cache, h: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        m, o = lw.spec.mixer, lw.offs
        proj, dt = ops.linear(h, lw.w_in), ops.linear(h, lw.w_step, epi=ops.EPI_F32)
        x = self._convolve(lw, cache, proj[:, o["x"]:], fb)
        y = ops.state_space(x, (0, o["B"] - o["x"], o["C"] - o["x"]), m.heads, m.groups, m.state, m.vdim, dt, lw.dt_bias, lw.A_log,
                            lw.D, cache.rec_state, fb.positions, fb.seq_cu, fb.seq_slots, fb.num_prefill_seqs)
        rows = torch.empty((h.shape[0], lw.w_o.shape[1]), dtype=h.dtype, device=h.device)
        ops.gated_norm_rows(y, proj[:, o["z"]:o["z"] + m.out_width], lw.head_norm, m.norm_groups, self.cfg.rms_norm_eps, rows)
        return ops.linear(rows, lw.w_o)

    def _parallel(self, lw: PreNormLayer, cache, h: torch.Tensor, fb: ForwardBatch) -> tuple:
        """Outputs of the two mixers, not yet normed."""
        a, b, o, T = lw.spec.mixer.left, lw.spec.mixer.right, lw.offs, h.shape[0]
        proj, beta = ops.linear(h, lw.w_in), ops.linear(h, lw.w_step, epi=ops.EPI_F32)

        def part(name, width):
            return proj[:, o[name]:o[name] + width]

        heads = self._attend(lw, a, tuple(o["left." + n] for n in "qkv"), cache, proj, fb)
        rows = torch.empty((T, lw.w_o.shape[1]), dtype=h.dtype, device=h.device)
        ops.gated_rows(heads, a.vdim, part("left.g", a.out_width), rows)
        left = ops.linear(rows, lw.w_o)

        x = self._convolve(lw, cache, part("right.q", b.channels), fb)
        decay = ops.linear(part("right.a1", lw.w_decay.shape[1]), lw.w_decay, epi=ops.EPI_F32)
        start = o["right.q"]
        heads = ops.delta_rule(x, tuple(o["right." + n] - start for n in "qkv"), b.heads, b.kv_heads, b.dim, b.vdim, decay,
                               lw.dt_bias, lw.A_log, beta, cache.rec_state, fb.positions, fb.seq_cu, fb.seq_slots,
                               fb.num_prefill_seqs, fb.num_prefill_tokens)
        gate = ops.linear(part("right.g1", lw.w_gate.shape[1]), lw.w_gate)
        rows = torch.empty((T, lw.w_o2.shape[1]), dtype=h.dtype, device=h.device)
        ops.gated_rows(heads, b.vdim, gate[:, :b.out_width], rows, lw.head_norm, self.cfg.rms_norm_eps, per_head=True)
        return left, ops.linear(rows, lw.w_o2)

    # ------------------------------------------------------------------ forward
    def forward_layers(self, x: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        eps, groups, v_first = self.cfg.rms_norm_eps, self.cfg.norm_groups, None
        if not self.is_first:
            x = x.clone()       # the residual is updated in place; the incoming buffer belongs to the caller
        h = ops.row_norm(x, self.layers[0].norm1, eps, ops.NORM_RMS, dtype=self.dtype, groups=groups)
        for li, lw in enumerate(self.layers):
            m, cache = lw.spec.mixer, self.kv_caches[li]
            leave = self.layers[li + 1].norm1 if li + 1 < len(self.layers) else None
            y = branches = None
            if isinstance(m, ParallelSpec):
                left, right = self._parallel(lw, cache, h, fb)
                branches = (m.left_scale, (left, lw.norm_left), (right, lw.norm_right))
            elif isinstance(m, StateSpaceSpec):
                y = self._state_space(lw, cache, h, fb)
            else:
                proj = ops.linear(h, lw.w_in, bias=lw.b_in)
                mixes = m.v_first is not None
                heads = self._attend(lw, m, tuple(lw.offs[n] for n in "qkv"), cache, proj, fb, v_first if mixes else None)
                if m.v_mix and not mixes:
                    v_first = proj[:, lw.offs["v"]:lw.offs["v"] + m.v_rows]
                y = ops.linear(heads.view(h.shape[0], -1), lw.w_o)
            h = ops.residual_add(x, y, leave if lw.moe is None else lw.norm2, eps, groups=groups, branches=branches)
            if lw.moe is not None:
                routed, _ = lw.moe.forward(h)
                h = ops.residual_add(x, None, leave, eps, routed, h, groups=groups)
        return x
