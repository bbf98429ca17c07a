"""Pipeline-stage model for decoders that list their layers one by one and mix tokens with windowed latent
attention (``Piburax``).

What differs from the MLA families of :mod:`parallax_b200.models.deepseek`, each a parameter of the layer or
of the op that runs it:

* every layer carries its own sizes (:class:`parallax_b200.models.layer_spec.LayerSpec`), also the widths of
  its cache rows;
* the residual is kept in fp32 (``hidden_dtype``) and sublayers are normed on their OUTPUT:
  ``x += residual_mult * norm(sublayer(x))`` (:func:`ops.residual_norm`, one kernel that also writes the
  low-precision copy of ``x`` the next projection reads);
* the embedding adds a hashed row of (previous token, token) (:func:`ops.embed_rows`; the batch brings the
  previous token of every row);
* attention sees a sliding window, its softmax has a learned sink per head, and the concatenated heads are
  gated by ``sigmoid(W_g x)`` - the gate rides in the epilogue of the value up-projection;
* the feed-forward is a clipped GLU, fused into the gate/up product's epilogue.

Attention runs in absorbed form over ``latent | rotated key`` cache rows for prompts and decoding alike.
One projection produces ``q | latent, key | gate`` (:attr:`LatentLayer.w_in`); the mixer is also that of
:mod:`parallax_b200.models.looped`, without a gate and with queries that go through a normed latent. The stage runs in bf16 (tensor
cores; fp32 where the design keeps fp32) or entirely in fp32 (``dtype=torch.float32``).
"""

from __future__ import annotations

import torch

from parallax_b200 import ops
from parallax_b200.engine.batch import ForwardBatch
from parallax_b200.models.layer_list import LayerListStage, ListedLayer, pad_rows


LATENT_SLOTS = ("w_in", "q_norm", "w_uq", "kv_norm", "w_uk_s", "w_uv", "sinks", "w_o")


def _up8(n: int) -> int:
    return n + -n % 8


def latent_shapes(m, width: int) -> dict[str, tuple]:
    """Checkpoint tensors of a latent-attention mixer (:class:`LatentAttentionSpec`)."""
    sh = {"dkv": (m.row_width, width), "dkv.norm": (m.kv_rank,), "uk": (m.heads * m.dim, m.kv_rank),
          "uv": (m.heads * m.vdim, m.kv_rank), "sink": (m.heads,), "o": (width, m.heads * m.vdim)}
    if m.q_rank:
        sh.update({"dq": (m.q_rank, width), "dq.norm": (m.q_rank,), "uq": (m.heads * m.q_width, m.q_rank)})
    else:
        sh["q"] = (m.heads * m.q_width, width)
    if m.gated:
        sh["g"] = (m.heads * m.vdim, width)
    return sh


def load_latent(lw, m, get) -> None:
    """Weights of a latent-attention mixer into a layer with :data:`LATENT_SLOTS`; ``get(name, dtype)``."""
    # the products that read x, one matrix: queries (or their latent) | latent and rotated key | output gate
    parts = ("dq" if m.q_rank else "q", "dkv") + (("g",) if m.gated else ())
    lw.w_in = torch.cat([pad_rows(get(n), 8) for n in parts], 0).contiguous()
    lw.q_norm = get("dq.norm", torch.float32) if m.q_rank else None
    lw.w_uq = pad_rows(get("uq"), 8) if m.q_rank else None
    lw.kv_norm = get("dkv.norm", torch.float32)
    # score = (W_uk^T q) . c: the key up-projection acts on the query
    lw.w_uk_s = get("uk").view(m.heads, m.dim, m.kv_rank).transpose(1, 2).reshape(-1, m.dim).contiguous()
    lw.w_uv = get("uv")
    lw.sinks = get("sink", torch.float32)
    lw.w_o = get("o")


def latent_mix(lw, m, cache: torch.Tensor, xl: torch.Tensor, fb: ForwardBatch, eps: float) -> torch.Tensor:
    """Output of a latent-attention mixer for the rows ``xl``; ``cache`` are its pages."""
    T, L, R = xl.shape[0], m.kv_rank, m.rot_dim
    proj = ops.linear(xl, lw.w_in)
    q_cat = torch.empty((T, m.heads, m.row_width), dtype=xl.dtype, device=xl.device)
    if m.q_rank:
        kv_off = _up8(m.q_rank)
        c_q = torch.empty((T, m.q_rank), dtype=xl.dtype, device=xl.device)
        ops.latent_rows(proj, 0, lw.q_norm, c_q, kv_off, lw.kv_norm, lw.cos_sin, fb.positions, fb.slot_mapping, cache, eps, L, R,
                        m.rot.dims)
        q = ops.linear(c_q, lw.w_uq)
        ops.latent_queries(q, m.heads, m.q_width, m.dim, lw.cos_sin, fb.positions, q_cat, L, R, m.rot.dims)
    else:
        kv_off, q = _up8(m.heads * m.q_width), proj
        ops.latent_prep(proj, kv_off, m.heads, m.q_width, m.dim, lw.kv_norm, lw.cos_sin, fb.positions, fb.slot_mapping, cache,
                        q_cat, eps, L, R, m.rot.dims)
    ops.head_linear(q, m.q_width, lw.w_uk_s, m.heads, q_cat[:, :, :L])
    o_lat = torch.empty((T, m.heads, L), dtype=xl.dtype, device=xl.device)
    Tp = fb.num_prefill_tokens
    if Tp:
        ops.latent_attn(q_cat[:Tp], cache, fb.p_block_tables, fb.p_cu_q, fb.p_ctx_lens, m.scale, L, m.window,
                        lw.sinks, fb.p_max_q, fb.p_max_ctx, out=o_lat[:Tp])
    if fb.num_decode:
        ops.latent_attn(q_cat[Tp:], cache, fb.d_block_tables, None, fb.d_ctx_lens, m.scale, L, m.window, lw.sinks,
                        1, fb.d_max_ctx, out=o_lat[Tp:])
    heads = torch.empty((T, m.heads, m.vdim), dtype=xl.dtype, device=xl.device)
    g_off = kv_off + _up8(m.row_width)
    ops.head_linear(o_lat.view(T, -1), L, lw.w_uv, m.heads, heads,
                    gate=proj[:, g_off:g_off + m.heads * m.vdim] if m.gated else None)
    return ops.linear(heads.view(T, -1), lw.w_o)


class LatentLayer(ListedLayer):
    __slots__ = LATENT_SLOTS + ("norm1", "norm2", "w_gu", "w_down", "moe")


class LatentStage(LayerListStage):
    layer_class = LatentLayer

    def __init__(self, *args, **kwargs):
        super().__init__(*args, **kwargs)
        # gate / up rows interleaved for the fused epilogue, or stacked for the separate activation kernel
        self.fused_glu = self.dtype == torch.bfloat16 and self.cfg.hidden_size % 8 == 0

    # ------------------------------------------------------------------ weights
    def weight_shapes(self, gi: int) -> dict[str, tuple]:
        """Checkpoint tensors of layer ``gi`` (name -> shape)."""
        W, spec = self.cfg.hidden_size, self.cfg.layer_specs[gi]
        p = f"l{gi}."
        sh = {p + "norm1": (W,), **{p + "mix." + n: s for n, s in latent_shapes(spec.mixer, W).items()}}
        if spec.mlp is not None:
            sh.update({p + "norm2": (W,), p + "mlp.gate": (spec.mlp.ff, W), p + "mlp.up": (spec.mlp.ff, W),
                       p + "mlp.down": (W, spec.mlp.ff)})
        return sh

    def _load_layer(self, lw: LatentLayer, gi: int, tensors) -> None:
        self._describe(lw, gi)
        spec, get = lw.spec, self._getter(gi, tensors)
        load_latent(lw, spec.mixer, lambda n, dt=self.dtype: get("mix." + n, dt))
        lw.norm1 = get("norm1", torch.float32)
        if spec.mlp is not None:
            lw.norm2 = get("norm2", torch.float32)
            if self.fused_glu:
                gate, up = pad_rows(get("mlp.gate"), 64), pad_rows(get("mlp.up"), 64)
                lw.w_gu = ops.interleave_gate_up(gate, up)
            else:
                gate, up = pad_rows(get("mlp.gate"), 8), pad_rows(get("mlp.up"), 8)
                lw.w_gu = torch.cat([gate, up], 0)
            # padded rows give activations of zero; the down projection gets zero columns for them
            down = get("mlp.down")
            lw.w_down = torch.nn.functional.pad(down, (0, gate.shape[0] - spec.mlp.ff)).contiguous()

    # ------------------------------------------------------------------ forward
    def _mixer(self, lw: LatentLayer, li: int, xl: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        return latent_mix(lw, lw.spec.mixer, self.kv_caches[li].k, xl, fb, self.cfg.rms_norm_eps)

    def _feed_forward(self, lw: LatentLayer, xl: torch.Tensor) -> torch.Tensor:
        limit = lw.spec.mlp.limit
        if self.fused_glu:
            act = ops.linear(xl, lw.w_gu, epi=ops.EPI_CLIP_GLU, limit=limit)
        else:
            act = ops.act_mul(ops.linear(xl, lw.w_gu), 1, limit)
        return ops.linear(act, lw.w_down)

    def forward_layers(self, h: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        eps, mult = self.cfg.rms_norm_eps, self.cfg.residual_mult
        if not self.is_first:
            h = h.clone()       # the residual is updated in place; the incoming buffer belongs to the caller
        xl = ops.to_low(h, self.dtype)
        for li, lw in enumerate(self.layers):
            xl = ops.residual_norm(h, self._mixer(lw, li, xl, fb), lw.norm1, eps, mult)
            if lw.spec.mlp is not None:
                xl = ops.residual_norm(h, self._feed_forward(lw, xl), lw.norm2, eps, mult)
        return h
