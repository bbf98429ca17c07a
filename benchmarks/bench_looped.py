"""Looped decoder (Zasalix) beside the closest other models of the framework at equal sizes: prefill and decode throughput of
a stack of layers, and every kernel of one layer against its roofline.

    python bench.py --design zasalix [--design-sizes 1b,8b]        (one JSON line)
    python benchmarks/bench_looped.py [--sizes 1b,8b] [--out FILE]

Three kinds of layers, each against its like: query-latent attention + dense feed-forward beside Piburax (latent attention
without a window + clipped GLU); windowed attention with a matrix memory beside it + routed experts beside Zudepel's
attention + routed experts (which has no second mixer); matrix memory + routed experts beside lightning attention + routed
experts. Only Zasalix has norms on both sides of a sublayer and token inputs. Random weights; a pass over a looped layer
costs what the layer costs, so stacks are timed without the loop. Timing as in ``bench_latent.py`` (CUDA graphs of stacks
larger than L2; single kernels with an L2 flush before every launch).
"""

from __future__ import annotations

import argparse
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

from benchmarks.bench_kernels import peaks  # noqa: E402
from benchmarks.bench_latent import Stack, kernel_rows, keys_seen  # noqa: E402
from benchmarks.bench_parallel_block import Rows, attention_rows as zudepel_attention_rows  # noqa: E402
from parallax_b200.models.config import config_from_hf, named_config  # noqa: E402
from parallax_b200.models.layer_spec import ACT_GELU_TANH, ParallelSpec  # noqa: E402
from parallax_b200.ops import cuda as cu  # noqa: E402

LAYERS = {"1b": 6, "8b": 3}
KINDS = ("latent_attention", "parallel", "mlstm")


def cut(cfg, kind: str, layers: int):
    """``layers`` copies of the first layer of a type, without the loop."""
    entry = next(e for e in cfg.raw["layers"] if e["type"] == kind)
    return config_from_hf(dict(cfg.raw, vocab=1024, layers=[entry] * layers, loop=None))


def twin_of(cfg, kind: str, layers: int):
    """(name, config) of the closest other design with the same sizes."""
    entry = next(e for e in cfg.raw["layers"] if e["type"] == kind)
    m, mlp = entry["mixer"], entry["mlp"]
    base = dict(vocab=1024, width=cfg.hidden_size, norm=dict(eps=1e-6))
    if kind == "latent_attention":
        mixer = {k: m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot")}
        layer = dict(type=kind, mixer=mixer, mlp=dict(kind="dense", ff=mlp["ff"], limit=6.0))
        return "piburax twin", config_from_hf(dict(base, architecture="Piburax", layers=[layer] * layers))
    if kind == "parallel":
        mixer = {k: m["left"][k] for k in ("heads", "kv_heads", "dim", "vdim", "scale", "rot")}
        layer = dict(type="attention", mixer=dict(mixer, conv=4), mlp=mlp)
    else:
        layer = dict(type="lightning", mlp=mlp, mixer=dict(heads=m["heads"], dim=m["dim"], vdim=m["vdim"],
                                                           decay=[1 - 2.0 ** -(1 + j % 10) for j in range(m["heads"])]))
    return "zudepel twin", config_from_hf(dict(base, architecture="Zudepel", layers=[layer] * layers))


# ---------------------------------------------------------------------------------- kernels of one layer
def norm_bytes(T: int, W: int, reads: float = 2.0, writes: float = 2.0) -> float:
    """Residual read and written in fp32, ``reads`` / ``writes`` further bytes per element."""
    return T * W * (8.0 + reads + writes)


def routed_rows(r: Rows, lw, x) -> None:
    s, moe, T, W = lw.spec.mlp, lw.moe, x.shape[0], x.shape[1]
    E, zudepel = s.experts, s.correction
    r.add("router", lambda: cu.linear(x, moe.router, epi=cu.EPI_F32), 2.0 * T * W * moe.router.shape[0],
          2.0 * (T * W + moe.router.numel()) + 4.0 * T * moe.router.shape[0])
    logits = cu.linear(x, moe.router, epi=cu.EPI_F32)

    def pick():
        return cu.moe_route(logits[:, :E], moe.correction, s.top, int(s.sigmoid), s.normalised)

    r.add("choice of experts", pick, 0, T * (4.0 * E + 8.0 * s.top))
    ids, wts = pick()
    plan = cu.moe_align(ids, E)
    pairs, n1, n2, k2 = ids.numel(), moe.w1.shape[0] // E, moe.w2.shape[0] // E, moe.w2.shape[1]
    used = int((torch.bincount(ids.long().flatten(), minlength=E) > 0).sum())
    r.add("expert lists", lambda: cu.moe_align(ids, E), 0, 16.0 * pairs)
    spread = (lambda: cu.moe_gather(x, plan)) if zudepel else (lambda: cu.moe_scatter_rows(x, plan, wts))
    # (a gather reads each pair's row; with the weights in it every token is read once)
    r.add("rows in expert order" + ("" if zudepel else ", weighted"), spread, 0, 2.0 * pairs * W + 2.0 * (pairs if zudepel else T) * W)
    xp = spread()
    r.add("experts: gate / up (+ SiLU)", lambda: cu.grouped_linear(xp, moe.w1, plan, E, epi=cu.EPI_SILU_MUL),
          2.0 * pairs * n1 * W, 2.0 * (pairs * (W + n1 / 2) + used * n1 * W))
    act = cu.grouped_linear(xp, moe.w1, plan, E, epi=cu.EPI_SILU_MUL)
    r.add("experts: down", lambda: cu.grouped_linear(act, moe.w2, plan, E), 2.0 * pairs * n2 * k2,
          2.0 * (pairs * (k2 + n2) + used * n2 * k2))
    return cu.grouped_linear(act, moe.w2, plan, E), plan, pairs, wts


def zasalix_rows(r: Rows, keys: int, kv_tokens: int) -> None:
    st, fb, T = r.stack.stage, r.fb, r.fb.num_tokens
    lw, lc, W, dev = st.layers[0], r.stack.pool.layers[0], r.stack.cfg.hidden_size, r.stack.dev
    m, mlp, x, h = lw.spec.mixer, lw.spec.mlp, r.rnd(T, W), torch.randn(T, W, device=r.stack.dev)
    empty = lambda *s: torch.empty(s, dtype=torch.bfloat16, device=dev)  # noqa: E731
    if hasattr(m, "kv_rank"):
        H, L, R, Q = m.heads, m.kv_rank, m.rot_dim, m.q_rank
        r.gemm("query latent | latent projection", x, lw.w_in)
        proj, c_q, q_cat = cu.linear(x, lw.w_in), empty(T, Q), empty(T, H, L + R)
        r.add("cache rows, norm of the query latent", lambda: cu.latent_rows(
            proj, 0, lw.q_norm, c_q, Q, lw.kv_norm, lw.cos_sin, fb.positions, fb.slot_mapping, lc.k, 1e-6, L, R, R), 0,
            4.0 * T * (L + R + Q))
        r.gemm("q projection", c_q, lw.w_uq)
        q = cu.linear(c_q, lw.w_uq)
        r.add("query rotation", lambda: cu.latent_queries(q, H, m.q_width, m.dim, lw.cos_sin, fb.positions, q_cat, L, R, R), 0,
              4.0 * T * H * R)
        r.add("key up-projection of q", lambda: cu.head_linear(q, m.q_width, lw.w_uk_s, H, q_cat[:, :, :L]),
              2.0 * T * H * L * m.dim, 2.0 * (T * H * (m.dim + L) + H * L * m.dim))
        o_lat = empty(T, H, L)
        bt, cq, ctx, mq, mc = (fb.p_block_tables, fb.p_cu_q, fb.p_ctx_lens, fb.p_max_q, fb.p_max_ctx) if fb.num_prefill_tokens \
            else (fb.d_block_tables, None, fb.d_ctx_lens, 1, fb.d_max_ctx)
        r.add("attention", lambda: cu.latent_attn(q_cat, lc.k, bt, cq, ctx, m.scale, L, 0, lw.sinks, mq, mc, out=o_lat),
              2.0 * keys * H * (2 * L + R), 2.0 * (kv_tokens * (L + R) + T * H * (2 * L + R)))
        heads = empty(T, H, m.vdim)
        r.add("value up-projection", lambda: cu.head_linear(o_lat.view(T, -1), L, lw.w_uv, H, heads),
              2.0 * T * H * L * m.vdim, 2.0 * (T * H * (m.vdim + L) + H * L * m.vdim))
        r.gemm("output projection", r.rnd(T, H * m.vdim), lw.w_o)
    else:
        both = isinstance(m, ParallelSpec)
        mem, p, o = (m.right, "right.", lw.offs) if both else (m, "", lw.offs)
        r.gemm("input projection", x, lw.w_in)
        proj, cat, at = cu.linear(x, lw.w_in), empty(T, lw.w_o.shape[1]), 0
        r.add("gates of the memory", lambda: cu.linear(x, lw.w_gates, epi=cu.EPI_F32), 2.0 * T * W * lw.w_gates.shape[0],
              2.0 * (T * W + lw.w_gates.numel()) + 4.0 * T * lw.w_gates.shape[0])
        gates = cu.linear(x, lw.w_gates, epi=cu.EPI_F32)
        if both:
            a = m.left
            q, offs = empty(T, a.heads, a.head_cols), tuple(o["left." + n] for n in "qkv")
            r.add("rotation, cache", lambda: cu.conv_qkv_prep(
                proj, offs, a.heads, a.kv_heads, a.dim, a.vdim, None, None, None, None, lw.cos_sin, fb.positions, fb.seq_cu,
                fb.seq_slots, fb.num_prefill_seqs, fb.num_prefill_tokens, fb.slot_mapping, lc.k, lc.v, q, 0.0), 0,
                4.0 * T * (a.q_rows + a.k_rows + a.v_rows))

            def attend():
                if fb.num_prefill_tokens:
                    return cu.attn_prefill(q, lc.k, lc.v, fb.p_block_tables, fb.p_cu_q, fb.p_ctx_lens, fb.p_max_q, a.scale,
                                           window=a.window, keep_first=a.keep_first)
                return cu.attn_decode(q, lc.k, lc.v, fb.d_block_tables, fb.d_ctx_lens, a.scale, window=a.window,
                                      max_ctx=fb.d_max_ctx, keep_first=a.keep_first)

            r.add("attention", attend, 4.0 * keys * a.heads * a.dim,
                  4.0 * (kv_tokens * a.kv_heads * a.dim + T * a.heads * a.dim))
            heads, at = attend(), a.out_width
            r.add("gate of the heads", lambda: cu.gated_rows(heads, a.vdim, proj[:, o["left.g"]:o["left.g"] + at], cat[:, :at],
                                                             scale=0.5), 0, 6.0 * T * at)
        seqs = fb.seq_slots.numel()

        def remember():
            return cu.matrix_memory(proj, tuple(o[p + n] for n in "qkv"), mem.heads, mem.dim, mem.vdim, gates, lw.b_gates,
                                    mem.gate_cap, lc.rec_state, fb.positions, fb.seq_cu, fb.seq_slots, fb.num_prefill_seqs)

        carried = 4.0 * (2 if fb.num_decode else 1) * seqs * mem.heads * mem.dim * mem.vdim
        r.add("linear attention", remember, 4.0 * T * mem.heads * mem.dim * mem.vdim,
              4.0 * T * mem.heads * (mem.dim + mem.vdim) + carried)
        mh, g0 = remember(), o[p + "g"]
        r.add("norm + gate of the heads", lambda: cu.gated_rows(mh, mem.vdim, proj[:, g0:g0 + mem.out_width], cat[:, at:],
                                                                lw.mem_norm, 1e-6, per_head=True, scale=0.5), 0,
              6.0 * T * mem.out_width)
        r.gemm("output projection", cat, lw.w_o)
    y = r.rnd(T, W)
    r.add("norm + residual + norm", lambda: cu.residual_step(h, y, lw.norm1b.args(), pre=lw.norm2.args(), dtype=torch.bfloat16), 0,
          norm_bytes(T, W))
    if lw.moe is None:
        r.gemm("up (+ activation)", x, lw.w_up, lambda: cu.act_linear(x, lw.w_up, mlp.act))
        r.gemm("down projection", r.rnd(T, lw.w_down.shape[1]), lw.w_down)
        routed, more = None, 0.0
    else:
        y2, plan, pairs, _ = routed_rows(r, lw, x)
        if mlp.shared:
            r.gemm("shared: gate / up (+ activation)", x, lw.w_gu, lambda: cu.glu_linear(x, lw.w_gu, mlp.shared.act), True)
            r.gemm("shared: down projection", r.rnd(T, lw.w_down.shape[1]), lw.w_down)
        routed, more = (y2, plan.pos_of, None), 2.0 * W * pairs
    name = "norm + residual" if routed is None else "experts' sum + norm + residual"
    r.add(name, lambda: cu.residual_step(h, y, lw.norm2b.args(), routed, pre=(), dtype=torch.bfloat16), 0,
          norm_bytes(T, W) + more)
    if not r.stack.cfg.token_side_dim:
        return
    r.gemm("token input: gate (+ activation, row)", x, lw.side_gate,
           lambda: cu.act_linear(x, lw.side_gate, ACT_GELU_TANH, st.side_table, fb.input_ids, 0))
    g = cu.act_linear(x, lw.side_gate, ACT_GELU_TANH, st.side_table, fb.input_ids, 0)
    r.gemm("token input: projection", g, lw.side_proj)
    r.add("token input: norm + residual + norm",
          lambda: cu.residual_step(h, y, (lw.side_norm,), eps=1e-6, pre=lw.norm1.args(), dtype=torch.bfloat16), 0, norm_bytes(T, W))


def lightning_rows(r: Rows) -> None:
    st, fb, T = r.stack.stage, r.fb, r.fb.num_tokens
    lw, W = st.layers[0], r.stack.cfg.hidden_size
    m, o, mlp = lw.spec.mixer, lw.offs, lw.spec.mlp
    x, seqs = r.rnd(T, W), fb.seq_slots.numel()
    r.gemm("input projection", x, lw.w_in)
    proj, state = cu.linear(x, lw.w_in), r.stack.pool.layers[0].rec_state

    def mix():
        return cu.lightning_attn(proj, (o["q"], o["k"], o["v"]), m.heads, m.dim, m.vdim, lw.decay_pow, state, fb.positions,
                                 fb.seq_cu, fb.seq_slots, fb.num_prefill_seqs)

    carried = 4.0 * (2 if fb.num_decode else 1) * seqs * m.heads * m.dim * m.vdim
    r.add("linear attention", mix, 4.0 * T * m.heads * m.dim * m.vdim, 4.0 * T * m.heads * (m.dim + m.vdim) + carried)
    heads, cat = mix(), r.rnd(T, lw.w_out.shape[1])
    r.add("norm + gate of the heads", lambda: cu.gated_rows(heads, m.vdim, proj[:, o["g"]:o["g"] + m.out_width],
                                                            cat[:, :m.out_width], lw.mix_norm, 1e-6), 0, 6.0 * T * m.out_width)
    y2, plan, pairs, wts = routed_rows(r, lw, x)
    gate = torch.zeros(T, device=x.device)
    if mlp.shared:
        r.gemm("shared: gate / up (+ activation)", x, lw.w_gu, lambda: cu.glu_linear(x, lw.w_gu, mlp.shared.act, gate,
                                                                                     cat[:, m.out_width:]), True)
    r.gemm("output + shared down projection" if mlp.shared else "output projection", cat, lw.w_out)
    h, y = torch.randn(T, W, device=r.stack.dev), r.rnd(T, W)
    r.add("experts' sum + residual + norm", lambda: cu.residual_add(h, y, lw.norm1, 1e-6, (y2, plan.pos_of, wts), x), 0,
          norm_bytes(T, W) + 2.0 * W * pairs)


BATCHES = (("prefill 1 x 1024", [1024], []), ("prefill 1 x 4096", [4096], []), ("prefill 8 x 512", [512] * 8, []),
           ("decode 1 x 1024", [], [1024]), ("decode 32 x 1024", [], [1024] * 32), ("decode 128 x 2048", [], [2048] * 128))
TIMED = ("prefill 1 x 4096", "decode 32 x 1024", "decode 128 x 2048")      # batches whose kernels are timed alone


def run(sizes: list, log=print) -> dict:
    table, kernels = [], []
    peaks()
    for size in sizes:
        base, n = named_config(f"zasalix-{size}"), LAYERS[size]
        for kind in KINDS:
            for name, cfg in (("zasalix", cut(base, kind, n)), twin_of(base, kind, n)):
                st = Stack(cfg, 264 * 1024)
                for label, prefill, decode in BATCHES:
                    fb = st.batch(prefill, decode)
                    fb.input_ids.copy_(torch.randint(0, 1024, (fb.num_tokens,), device=st.dev))
                    ms = st.time(fb)
                    table.append(dict(size=size, layer=kind, model=name, batch=label, layers=n, ms_per_layer=round(ms / n, 4),
                                      tokens_per_s_per_layer=round(fb.num_tokens / (ms / n) * 1e3)))
                    log(table[-1])
                    if size != sizes[-1] or label not in TIMED:
                        continue
                    spec = cfg.layer_specs[0].mixer
                    win = spec.window if name == "zasalix" and kind == "parallel" else 0
                    keep = spec.left.keep_first if win else 0
                    keys = sum(keys_seen(p, win) + sum(min(keep, max(i - win + 1, 0)) for i in range(p) if win) for p in prefill)
                    keys += sum(min(c, win + keep) if win else c for c in decode)
                    kv = sum(prefill) + sum(min(c, win + keep) if win else c for c in decode)
                    r = Rows(st, fb, label)
                    if name == "zasalix":
                        zasalix_rows(r, keys, kv)
                    elif kind == "latent_attention":
                        r.rows = kernel_rows(st, fb, label, keys, kv)
                    elif kind == "parallel":
                        zudepel_attention_rows(r, keys, kv)
                    else:
                        lightning_rows(r)
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
