"""Pre-norm decoder with three kinds of mixers (Kikurax) beside the closest other models of the framework at equal sizes: prefill
and decode throughput of a stack of layers, and every kernel of one layer against its roofline.

    python bench.py --design kikurax [--design-sizes 1b,8b]        (one JSON line)
    python benchmarks/bench_prenorm.py [--sizes 1b,8b] [--out FILE]

Three kinds of layers, each with routed experts, against its like: soft-capped attention beside Zudepel's attention (which has
a convolution and an output gate, and no cap); a state-space layer beside lightning attention with the same state and output
width (whose q and k are not shared by groups, and which has no convolution); sigmoid attention with a gated delta rule beside
it next to Zasalix's attention with a matrix memory beside it. The kernels of a Qwen3-Next-style gated delta net of the same
heads are listed as well. Random weights. Timing as in ``bench_latent.py`` (CUDA graphs of stacks larger than L2; single
kernels with an L2 flush before every launch).
"""

from __future__ import annotations

import argparse
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

from benchmarks import bench_looped, bench_parallel_block  # noqa: E402
from benchmarks.bench_kernels import peaks  # noqa: E402
from benchmarks.bench_latent import Stack, keys_seen  # noqa: E402
from benchmarks.bench_parallel_block import BATCHES, TIMED, Rows  # noqa: E402
from parallax_b200.models.config import config_from_hf, named_config  # noqa: E402
from parallax_b200.models.layer_spec import ParallelSpec, StateSpaceSpec  # noqa: E402
from parallax_b200.ops import cuda as cu  # noqa: E402

LAYERS = {"1b": 6, "8b": 3}
KINDS = ("attention", "mamba2", "parallel")


def cut(cfg, kind: str, layers: int):
    """``layers`` copies of the first layer of a type."""
    entry = next(e for e in cfg.raw["layers"] if e["type"] == kind)
    return config_from_hf(dict(cfg.raw, vocab=1024, layers=[entry] * layers))


def twin_of(cfg, kind: str, layers: int):
    """(name, config) of the closest other design with the same sizes."""
    entry = next(e for e in cfg.raw["layers"] if e["type"] == kind)
    m, mlp = entry["mixer"], dict(entry["mlp"], expert=dict(ff=entry["mlp"]["expert"]["ff"]))
    base, head = dict(vocab=1024, width=cfg.hidden_size, norm=dict(eps=1e-6)), ("heads", "kv_heads", "dim", "vdim", "scale")
    if kind == "attention":
        mixer = dict({k: m[k] for k in head}, conv=4, rot=dict(base=1e4, dims=m["rot"]["dims"]))
        layer, arch = dict(type="attention", mixer=mixer, mlp=mlp), "Zudepel"
    elif kind == "mamba2":
        h = m["heads"] * m["vdim"] // m["state"]
        mixer = dict(heads=h, dim=m["state"], vdim=m["state"], decay=[1 - 2.0 ** -(1 + j % 10) for j in range(h)])
        layer, arch = dict(type="lightning", mixer=mixer, mlp=mlp), "Zudepel"
    else:
        a, b = m["left"], m["right"]
        left = dict({k: a[k] for k in head}, rot=dict(base=1e4, dims=a["dim"]))
        right = dict(heads=b["heads"], dim=b["dim"], vdim=b["vdim"], gate_cap=15.0)
        layer, arch = dict(type="parallel", mixer=dict(left=left, right=right, left_scale=0.5, right_scale=0.5), mlp=mlp), "Zasalix"
    return f"{arch.lower()} twin", config_from_hf(dict(base, architecture=arch, layers=[layer] * layers))


# ---------------------------------------------------------------------------------- kernels of one layer
def kikurax_rows(r: Rows, keys: int, kv_tokens: int) -> None:
    st, fb, T = r.stack.stage, r.fb, r.fb.num_tokens
    lw, lc, W, dev, o = st.layers[0], r.stack.pool.layers[0], r.stack.cfg.hidden_size, r.stack.dev, st.layers[0].offs
    m, s, moe, groups = lw.spec.mixer, lw.spec.mlp, lw.moe, r.stack.cfg.norm_groups
    x, h, seqs = r.rnd(T, W), torch.randn(T, W, device=dev), fb.seq_slots.numel()
    empty = lambda *sh: torch.empty(sh, dtype=torch.bfloat16, device=dev)  # noqa: E731
    runs = (fb.positions, fb.seq_cu, fb.seq_slots, fb.num_prefill_seqs)
    r.gemm("input projection", x, lw.w_in, lambda: cu.linear(x, lw.w_in, bias=lw.b_in))
    proj = cu.linear(x, lw.w_in, bias=lw.b_in)

    def thin(name, a, w, f32=True):
        r.add(name, lambda: cu.linear(a, w, epi=cu.EPI_F32 if f32 else cu.EPI_NONE), 2.0 * T * w.numel(),
              2.0 * (T * w.shape[1] + w.numel()) + (4.0 if f32 else 2.0) * T * w.shape[0])
        return cu.linear(a, w, epi=cu.EPI_F32 if f32 else cu.EPI_NONE)

    def attend(a, offs):
        q = empty(T, a.heads, a.head_cols)
        r.add("norm, rotation, cache", lambda: cu.head_qkv_prep(
            proj, offs, a.heads, a.kv_heads, a.dim, a.vdim, 1e-6, lw.cos_sin, fb.positions, fb.slot_mapping, lc.k, lc.v, q,
            lw.head_scale, lw.pos_scale), 0, 4.0 * T * (a.q_rows + a.k_rows + a.v_rows))
        kw = dict(sinks=lw.sinks, softcap=a.softcap, sigmoid_bias=lw.sig_bias)

        def fn():
            if fb.num_prefill_tokens:
                return cu.attn_prefill(q, lc.k, lc.v, fb.p_block_tables, fb.p_cu_q, fb.p_ctx_lens, fb.p_max_q, a.scale, **kw)
            return cu.attn_decode(q, lc.k, lc.v, fb.d_block_tables, fb.d_ctx_lens, a.scale, max_ctx=fb.d_max_ctx, **kw)

        r.add("attention", fn, 4.0 * keys * a.heads * a.dim, 4.0 * (kv_tokens * a.kv_heads * a.dim + T * a.heads * a.dim))
        return fn()

    def convolve(cols, taps):
        def fn():
            return cu.short_conv(cols, lw.conv_w, lw.conv_b, lc.conv_state, *runs, fb.num_prefill_tokens)

        C = cols.shape[1]
        r.add("convolution", fn, 0, 4.0 * T * C + (4.0 * (taps - 1) * T * C if fb.num_decode else 0))
        return fn()

    def carried(heads, dk, dv):
        return 4.0 * (2 if fb.num_decode else 1) * seqs * heads * dk * dv

    y, branches = r.rnd(T, W), None
    if isinstance(m, StateSpaceSpec):
        dt = thin("step sizes", x, lw.w_step)
        c = convolve(proj[:, o["x"]:], m.conv)

        def scan():
            return cu.state_space(c, (0, o["B"] - o["x"], o["C"] - o["x"]), m.heads, m.groups, m.state, m.vdim, dt, lw.dt_bias,
                                  lw.A_log, lw.D, lc.rec_state, *runs)

        r.add("linear attention", scan, 4.0 * T * m.heads * m.state * m.vdim,
              4.0 * T * (m.out_width + m.bc_rows) + carried(m.heads, m.state, m.vdim))
        heads, rows = scan(), empty(T, lw.w_o.shape[1])
        r.add("norm + gate of the heads", lambda: cu.gated_norm_rows(heads, proj[:, :m.out_width], lw.head_norm, m.norm_groups, 1e-6,
                                                                     rows), 0, 6.0 * T * m.out_width)
        r.gemm("output projection", rows, lw.w_o)
    elif isinstance(m, ParallelSpec):
        a, b = m.left, m.right
        heads = attend(a, tuple(o["left." + n] for n in "qkv"))
        rows = empty(T, lw.w_o.shape[1])
        r.add("gate of the heads", lambda: cu.gated_rows(heads, a.vdim, proj[:, o["left.g"]:o["left.g"] + a.out_width], rows), 0,
              6.0 * T * a.out_width)
        r.gemm("output projection", rows, lw.w_o)
        beta = thin("gates of the memory", x, lw.w_step)
        start = o["right.q"]
        c = convolve(proj[:, start:start + b.channels], b.conv)
        decay = thin("decays", proj[:, o["right.a1"]:o["right.a1"] + lw.w_decay.shape[1]], lw.w_decay)

        def scan():
            return cu.delta_rule(c, tuple(o["right." + n] - start for n in "qkv"), b.heads, b.kv_heads, b.dim, b.vdim, decay,
                                 lw.dt_bias, lw.A_log, beta, lc.rec_state, *runs, fb.num_prefill_tokens)

        r.add("linear attention", scan, 6.0 * T * b.heads * b.dim * b.vdim,
              4.0 * T * b.heads * b.vdim + T * (4.0 * b.q_rows + 4.0 * b.heads * b.dim) + carried(b.heads, b.dim, b.vdim))
        mem = scan()
        gate = thin("gate projection", proj[:, o["right.g1"]:o["right.g1"] + lw.w_gate.shape[1]], lw.w_gate, False)
        rows2 = empty(T, lw.w_o2.shape[1])
        r.add("norm + gate of the heads", lambda: cu.gated_rows(mem, b.vdim, gate[:, :b.out_width], rows2, lw.head_norm, 1e-6,
                                                                per_head=True), 0, 6.0 * T * b.out_width)
        r.gemm("second output projection", rows2, lw.w_o2)
        branches = (0.5, (y, lw.norm_left), (r.rnd(T, W), lw.norm_right))
    else:
        heads = attend(m, tuple(o[n] for n in "qkv"))
        r.gemm("output projection", heads.view(T, -1), lw.w_o)
    r.add("norm + residual + norm" if branches else "residual + norm",
          lambda: cu.residual_add(h, None if branches else y, lw.norm2, 1e-6, groups=groups, branches=branches), 0,
          T * W * (14.0 if branches else 12.0))
    thin("router", x, moe.router)
    logits = cu.linear(x, moe.router, bias=moe.bias, epi=cu.EPI_F32)

    def pick():
        return cu.moe_route(logits[:, :s.outputs], None, s.top, 0, True)

    r.add("choice of experts", pick, 0, T * (4.0 * s.outputs + 8.0 * s.top))
    ids, wts = pick()
    y2, plan, pairs = r.experts(x, ids, moe.w1, moe.w2, s.experts, cu.EPI_CLIP_GLU, moe.limit)
    r.add("experts' sum + residual + norm",
          lambda: cu.residual_add(h, None, lw.norm1, 1e-6, (y2, plan.pos_of, wts), x, groups=groups), 0, T * W * 10.0 + 2.0 * W * pairs)


def run(sizes: list, log=print) -> dict:
    table, kernels = [], []
    peaks()
    for size in sizes:
        base, n = named_config(f"kikurax-{size}"), LAYERS[size]
        for kind in KINDS:
            models = [("kikurax", cut(base, kind, n)), twin_of(base, kind, n)]
            if kind == "parallel":
                b = base.layer_specs[0].mixer.right
                models.append(("delta net twin", config_from_hf(dict(
                    architectures=["Qwen3NextForCausalLM"], model_type="qwen3_next", hidden_size=base.hidden_size, num_hidden_layers=1,
                    num_attention_heads=8, num_key_value_heads=2, head_dim=128, intermediate_size=1024, vocab_size=1024,
                    rope_theta=1e4, max_position_embeddings=16384, linear_num_key_heads=b.kv_heads, linear_num_value_heads=b.heads,
                    linear_key_head_dim=b.dim, linear_value_head_dim=b.vdim, linear_conv_kernel_dim=4,
                    layer_types=["linear_attention"]))))
            for name, cfg in models:
                st = Stack(cfg, 264 * 1024)
                for label, prefill, decode in BATCHES:
                    fb = st.batch(prefill, decode)
                    if name != "delta net twin":
                        ms = st.time(fb)
                        table.append(dict(size=size, layer=kind, model=name, batch=label, layers=n, ms_per_layer=round(ms / n, 4),
                                          tokens_per_s_per_layer=round(fb.num_tokens / (ms / n) * 1e3)))
                        log(table[-1])
                    if size != sizes[-1] or label not in TIMED:
                        continue
                    keys, kv = sum(keys_seen(p, 0) for p in prefill) + sum(decode), sum(prefill) + sum(decode)
                    r = Rows(st, fb, label)
                    if name == "kikurax":
                        kikurax_rows(r, keys, kv)
                    elif name == "delta net twin":
                        bench_parallel_block.twin_linear_rows(r)
                        r.rows = [row for row in r.rows if row["kernel"] in ("convolution", "linear attention")]
                    elif kind == "attention":
                        bench_parallel_block.attention_rows(r, keys, kv)
                    elif kind == "mamba2":
                        bench_looped.lightning_rows(r)
                    else:
                        bench_looped.zasalix_rows(r, keys, kv)
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
