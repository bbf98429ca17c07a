"""Parallel-block decoder (Zudepel) beside the closest other model of the framework, a Qwen3-Next-style hybrid of equal
sizes: prefill and decode throughput of a stack of layers, and every kernel of one layer against its roofline.

    python bench.py --design zudepel [--design-sizes 1b,8b]        (one JSON line)
    python benchmarks/bench_parallel_block.py [--sizes 1b,8b] [--out FILE]

Two kinds of layers, each against its like: lightning attention + dense feed-forward beside gated delta net + dense
feed-forward, and attention + routed experts beside gated attention + routed experts. Random weights; timing as in
``bench_latent.py`` (CUDA graphs of stacks larger than L2; single kernels with an L2 flush before every launch).
"""

from __future__ import annotations

import argparse
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

from benchmarks.bench_kernels import peaks, time_fn  # noqa: E402
from benchmarks.bench_latent import Stack, keys_seen  # noqa: E402
from parallax_b200.models.config import LINEAR, config_from_hf, named_config  # noqa: E402
from parallax_b200.ops import cuda as cu  # noqa: E402

LAYERS = {"1b": 8, "8b": 4}


def cut(cfg, kind: str, layers: int):
    """``layers`` copies of the first layer of a type."""
    entry = next(e for e in cfg.raw["layers"] if e["type"] == kind)
    return config_from_hf(dict(cfg.raw, vocab=1024, layers=[entry] * layers))


def twin_of(cfg, kind: str, layers: int):
    """Hybrid decoder of the same sizes: gated delta net + dense, or gated attention + experts."""
    att = next(s for s in cfg.layer_specs if s.mixer.kind == "attention")
    lin = next(s for s in cfg.layer_specs if s.mixer.kind == LINEAR)
    a, m, moe = att.mixer, lin.mixer, att.mlp
    d = dict(architectures=["Qwen3NextForCausalLM"], model_type="qwen3_next", hidden_size=cfg.hidden_size,
             num_hidden_layers=layers, num_attention_heads=a.heads, num_key_value_heads=a.kv_heads, head_dim=a.dim,
             intermediate_size=lin.mlp.ff, vocab_size=1024, rope_theta=1e4, max_position_embeddings=16384,
             linear_num_key_heads=m.heads, linear_num_value_heads=m.heads, linear_key_head_dim=m.dim,
             linear_value_head_dim=m.vdim, linear_conv_kernel_dim=4,
             layer_types=["linear_attention" if kind == "lightning" else "full_attention"] * layers)
    if kind == "attention":
        d.update(num_experts=moe.outputs, num_experts_per_tok=moe.top, moe_intermediate_size=moe.expert.ff,
                 shared_expert_intermediate_size=moe.shared.ff, norm_topk_prob=True)
    return config_from_hf(d)


class Rows:
    """Kernel timings of one batch with their roofline fractions."""

    def __init__(self, stack: Stack, fb, label: str):
        self.hbm, self.tf, _ = peaks()
        self.stack, self.fb, self.label, self.rows = stack, fb, label, []

    def rnd(self, *s):
        return (torch.randn(*s, device=self.stack.dev) * 0.3).to(torch.bfloat16)

    def add(self, name, fn, flops, byts):
        ms = time_fn(fn)
        t_f, t_b = flops / (self.tf * 1e9), byts / (self.hbm * 1e6)
        self.rows.append(dict(batch=self.label, kernel=name, us=round(ms * 1e3, 1), roofline_frac=round(max(t_f, t_b) / ms, 4),
                              bound="compute" if t_f > t_b else "memory"))

    def gemm(self, name, x, w, fn=None, halves=False):
        (M, K), N = x.shape, w.shape[0]
        fn = fn or (lambda: cu.linear(x, w))
        self.add(name, fn, 2.0 * M * N * K, 2.0 * (M * K + N * K + M * N // (2 if halves else 1)))

    def experts(self, x, ids, w1, w2, E, epi=cu.EPI_SILU_MUL, limit=0.0):
        plan = cu.moe_align(ids, E)
        pairs, n1, n2, K = int((plan.pos_of >= 0).sum()), w1.shape[0] // E, w2.shape[0] // E, w1.shape[1]
        used = int((torch.bincount(ids[ids < E].long().flatten(), minlength=E) > 0).sum())
        self.add("expert lists", lambda: cu.moe_align(ids, E), 0, 16.0 * ids.numel())
        self.add("rows in expert order", lambda: cu.moe_gather(x, plan), 0, 4.0 * pairs * K)
        xp = cu.moe_gather(x, plan)
        self.add("experts: gate / up (+ SiLU)", lambda: cu.grouped_linear(xp, w1, plan, E, epi=epi, limit=limit),
                 2.0 * pairs * n1 * K, 2.0 * (pairs * (K + n1 / 2) + used * n1 * K))
        act = cu.grouped_linear(xp, w1, plan, E, epi=epi, limit=limit)
        k2 = act.shape[1]
        self.add("experts: down", lambda: cu.grouped_linear(act, w2, plan, E), 2.0 * pairs * n2 * k2,
                 2.0 * (pairs * (k2 + n2) + used * n2 * k2))
        return cu.grouped_linear(act, w2, plan, E), plan, pairs

    def attention(self, q, kc, vc, keys, kv_tokens, scale, sinks=None):
        fb, T, H, D, G = self.fb, q.shape[0], q.shape[1], q.shape[2], kc.shape[1]

        def fn():
            if fb.num_prefill_tokens:
                return cu.attn_prefill(q, kc, vc, fb.p_block_tables, fb.p_cu_q, fb.p_ctx_lens, fb.p_max_q, scale, sinks=sinks)
            return cu.attn_decode(q, kc, vc, fb.d_block_tables, fb.d_ctx_lens, scale, sinks=sinks, max_ctx=fb.d_max_ctx)

        self.add("attention", fn, 4.0 * keys * H * D, 4.0 * (kv_tokens * G * D + T * H * D))
        return fn()


def lightning_rows(r: Rows) -> None:
    st, fb, T = r.stack.stage, r.fb, r.fb.num_tokens
    lw, W = st.layers[0], r.stack.cfg.hidden_size
    m, o = lw.spec.mixer, lw.offs
    x, seqs = r.rnd(T, W), fb.seq_slots.numel()
    r.gemm("input projection", x, lw.w_in)
    proj, state = cu.linear(x, lw.w_in), r.stack.pool.layers[0].rec_state

    def mix():
        return cu.lightning_attn(proj, (o["q"], o["k"], o["v"]), m.heads, m.dim, m.vdim, lw.decay_pow, state, fb.positions,
                                 fb.seq_cu, fb.seq_slots, fb.num_prefill_seqs)

    carried = 4.0 * (2 if fb.num_decode else 1) * seqs * m.heads * m.dim * m.vdim
    r.add("linear attention", mix, 4.0 * T * m.heads * m.dim * m.vdim, 4.0 * T * m.heads * (m.dim + m.vdim) + carried)
    heads, cat = mix(), r.rnd(T, lw.w_out.shape[1])
    gate = proj[:, o["g"]:o["g"] + m.out_width]
    r.add("norm + gate of the heads", lambda: cu.gated_rows(heads, m.vdim, gate, cat[:, :m.out_width], lw.mix_norm, 1e-6), 0,
          6.0 * T * m.out_width)
    r.gemm("gate / up (+ activation)", x, lw.w_gu, lambda: cu.glu_linear(x, lw.w_gu, 2, None, cat[:, m.out_width:]), True)
    r.gemm("output + down projection", cat, lw.w_out)
    h, y = torch.randn(T, W, device=r.stack.dev), r.rnd(T, W)
    r.add("residual + norm", lambda: cu.residual_add(h, y, lw.norm1, 1e-6), 0, T * W * 12.0)


def attention_rows(r: Rows, keys: int, kv_tokens: int) -> None:
    st, fb, T = r.stack.stage, r.fb, r.fb.num_tokens
    lw, W, lc = st.layers[0], r.stack.cfg.hidden_size, r.stack.pool.layers[0]
    m, o, s, moe = lw.spec.mixer, lw.offs, lw.spec.mlp, lw.moe
    x = r.rnd(T, W)
    r.gemm("input projection", x, lw.w_in, lambda: cu.linear(x, lw.w_in, bias=lw.b_in))
    proj = cu.linear(x, lw.w_in, bias=lw.b_in)
    q = torch.empty((T, m.heads, m.head_cols), dtype=x.dtype, device=x.device)
    C = m.q_rows + m.k_rows + m.v_rows
    r.add("convolution, norm, rotation, cache",
          lambda: cu.conv_qkv_prep(proj, (o["q"], o["k"], o["v"]), m.heads, m.kv_heads, m.dim, m.vdim, lw.conv_w, lc.conv_state,
                                   lw.q_norm, lw.k_norm, lw.cos_sin, fb.positions, fb.seq_cu, fb.seq_slots, fb.num_prefill_seqs,
                                   fb.num_prefill_tokens, fb.slot_mapping, lc.k, lc.v, q, 1e-6),
          0, 4.0 * T * C + (4.0 * (m.conv - 1) * T * C if fb.num_decode else 0))
    heads = r.attention(q, lc.k, lc.v, keys, kv_tokens, m.scale, lw.sinks)
    cat, gate = r.rnd(T, lw.w_out.shape[1]), proj[:, o["g"]:o["g"] + m.out_width]
    r.add("gate of the heads", lambda: cu.gated_rows(heads, m.vdim, gate, cat[:, :m.out_width]), 0, 6.0 * T * m.out_width)
    r.add("router", lambda: cu.linear(x, moe.router, epi=cu.EPI_F32), 2.0 * T * W * moe.router.shape[0],
          2.0 * (T * W + moe.router.numel()) + 4.0 * T * moe.router.shape[0])
    logits = cu.linear(x, moe.router, epi=cu.EPI_F32)

    def pick():
        return cu.moe_route(logits[:, :s.outputs], moe.correction, s.top, 0, True, s.groups, s.groups_keep, group_top=1)

    r.add("choice of experts", pick, 0, T * (4.0 * s.outputs + 8.0 * s.top))
    ids, wts = pick()
    y2, plan, pairs = r.experts(x, ids, moe.w1, moe.w2, s.experts)
    if s.shared:
        r.gemm("shared: gate / up (+ activation)", x, lw.w_gu,
               lambda: cu.glu_linear(x, lw.w_gu, 0, logits[:, s.outputs], cat[:, m.out_width:]), True)
    r.gemm("output + shared down projection" if s.shared else "output projection", cat, lw.w_out)
    h, y = torch.randn(T, W, device=r.stack.dev), r.rnd(T, W)
    r.add("experts' sum + residual + norm", lambda: cu.residual_add(h, y, lw.norm1, 1e-6, (y2, plan.pos_of, wts), x), 0,
          T * W * 12.0 + 2.0 * W * (pairs + (T if pairs < T * s.top else 0)))


def twin_linear_rows(r: Rows) -> None:
    st, fb, T = r.stack.stage, r.fb, r.fb.num_tokens
    lw, W, lc = st.layers[0], r.stack.cfg.hidden_size, r.stack.pool.layers[0]
    Hk, Hv, Dk, Dv, n = st.Hk, st.Hv, st.Dk, st.Dv, st.qkv_dim
    x, seqs = r.rnd(T, W), fb.seq_slots.numel()
    r.gemm("input projection", x, lw.w_in)
    proj = cu.linear(x, lw.w_in)

    def conv():
        return cu.causal_conv1d_silu(proj[:, :n], lw.conv_w, lw.conv_b, lc.conv_state, fb.seq_cu, fb.seq_slots, fb.positions)

    r.add("convolution", conv, 0, 4.0 * T * n + (4.0 * 3 * T * n if fb.num_decode else 0))
    c, nz = conv(), Hv * Dv
    z, b, a = proj[:, n:n + nz], proj[:, n + nz:n + nz + Hv], proj[:, n + nz + Hv:n + nz + 2 * Hv]
    carried = 4.0 * (2 if fb.num_decode else 1) * seqs * Hv * Dk * Dv
    r.add("linear attention", lambda: cu.gated_delta_rule(c, a, b, lw.A_log, lw.dt_bias, z, lw.norm_w, lc.rec_state, fb.seq_cu,
                                                          fb.seq_slots, fb.positions, Hk, Hv, Dk, Dv, 1e-6),
          6.0 * T * Hv * Dk * Dv, 2.0 * T * (n + 2 * nz) + carried)
    heads, act = r.rnd(T, nz), r.rnd(T, lw.w_down.shape[1])
    r.gemm("output projection (+ residual)", heads, lw.w_out, lambda: cu.linear(heads, lw.w_out, residual=x))
    r.add("norm", lambda: cu.rmsnorm(x, lw.ln1, 1e-6), 0, T * W * 4.0)
    r.gemm("gate / up (+ activation)", x, lw.w_gu, lambda: cu.linear(x, lw.w_gu, epi=cu.EPI_SILU_MUL), True)
    r.gemm("down projection (+ residual)", act, lw.w_down, lambda: cu.linear(act, lw.w_down, residual=x))


def twin_attention_rows(r: Rows, keys: int, kv_tokens: int) -> None:
    st, fb, T = r.stack.stage, r.fb, r.fb.num_tokens
    lw, cfg, lc = st.layers[0], r.stack.cfg, r.stack.pool.layers[0]
    W, H, G, D, moe = cfg.hidden_size, cfg.num_attention_heads, cfg.num_key_value_heads, cfg.head_dim, lw.moe
    x = r.rnd(T, W)
    r.gemm("input projection", x, lw.w_qkv)
    qkv = cu.linear(x, lw.w_qkv)
    r.add("norm, rotation, cache",
          lambda: cu.qk_norm_rope_cache(qkv, lw.q_norm, lw.k_norm, st.cos_sin, fb.positions, fb.slot_mapping, lc.k, lc.v, H, G, D,
                                        cfg.rot_dim, 1e-6, 1.0), 0, 4.0 * qkv.numel())
    heads = r.attention(qkv.view(T, H + 2 * G, D)[:, :H], lc.k, lc.v, keys, kv_tokens, st.scale).view(T, H * D)
    r.gemm("gate projection", x, lw.w_gate)
    gate = cu.linear(x, lw.w_gate)
    r.add("gate of the heads", lambda: cu.sigmoid_gate_mul(heads, gate), 0, 6.0 * T * H * D)
    r.gemm("output projection (+ residual)", heads, lw.w_o, lambda: cu.linear(heads, lw.w_o, residual=x))
    r.add("norm", lambda: cu.rmsnorm(x, lw.ln1, 1e-6), 0, T * W * 4.0)
    r.add("router", lambda: cu.linear(x, moe.router, epi=cu.EPI_F32), 2.0 * T * W * moe.num_experts,
          2.0 * (T * W + moe.router.numel()) + 4.0 * T * moe.num_experts)
    logits = cu.linear(x, moe.router, epi=cu.EPI_F32)
    r.add("choice of experts", lambda: cu.moe_route(logits, None, moe.top_k), 0, T * (4.0 * moe.num_experts + 8.0 * moe.top_k))
    ids, wts = cu.moe_route(logits, None, moe.top_k)
    y2, plan, pairs = r.experts(x, ids, moe.w1, moe.w2, moe.num_experts)
    r.gemm("shared: gate / up (+ activation)", x, moe.shared_gu, lambda: cu.linear(x, moe.shared_gu, epi=cu.EPI_SILU_MUL), True)
    act = r.rnd(T, moe.shared_down.shape[1])
    r.gemm("shared: down (+ residual)", act, moe.shared_down, lambda: cu.linear(act, moe.shared_down, residual=x))
    r.add("experts' sum", lambda: cu.moe_combine(y2, plan, wts, x, T), 0, 4.0 * T * W + 2.0 * W * pairs)


BATCHES = (("prefill 1 x 1024", [1024], []), ("prefill 1 x 4096", [4096], []), ("prefill 8 x 512", [512] * 8, []),
           ("decode 1 x 1024", [], [1024]), ("decode 32 x 1024", [], [1024] * 32), ("decode 128 x 2048", [], [2048] * 128))
TIMED = ("prefill 1 x 4096", "decode 32 x 1024", "decode 128 x 2048")      # batches whose kernels are timed alone


def run(sizes: list, log=print) -> dict:
    table, kernels = [], []
    for size in sizes:
        base, n = named_config(f"zudepel-{size}"), LAYERS[size]
        for kind in ("lightning", "attention"):
            for name, cfg in (("zudepel", cut(base, kind, n)), ("hybrid twin", twin_of(base, kind, n))):
                st = Stack(cfg, 264 * 1024)
                for label, prefill, decode in BATCHES:
                    fb = st.batch(prefill, decode)
                    ms = st.time(fb)
                    table.append(dict(size=size, layer=kind, model=name, batch=label, layers=n, ms_per_layer=round(ms / n, 4),
                                      tokens_per_s_per_layer=round(fb.num_tokens / (ms / n) * 1e3)))
                    log(table[-1])
                    if size != sizes[-1] or label not in TIMED:
                        continue
                    r = Rows(st, fb, label)
                    if kind == "lightning":
                        (lightning_rows if name == "zudepel" else twin_linear_rows)(r)
                    else:
                        keys, kv = sum(keys_seen(p, 0) for p in prefill) + sum(decode), sum(prefill) + sum(decode)
                        (attention_rows if name == "zudepel" else twin_attention_rows)(r, keys, kv)
                    cu.check_status(st.dev)
                    for row in r.rows:
                        kernels.append(dict(size=size, layer=kind, model=name, **row))
                        log(kernels[-1])
                del st
                torch.cuda.empty_cache()
    return {"layers": table, "kernels": kernels}


def main(argv=None) -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="1b,8b")
    ap.add_argument("--out", default="")
    a = ap.parse_args(argv)
    res = run(a.sizes.split(","), log=lambda r: print(r, flush=True))
    if a.out:
        with open(a.out, "w") as f:
            json.dump(res, f, indent=1)


if __name__ == "__main__":
    main()
