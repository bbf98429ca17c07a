"""Windowed latent attention decoder (Piburax) beside the closest other model of the framework, a DeepSeek-style
MLA decoder with dense feed-forwards of equal sizes: prefill and decode throughput of a stack of layers, and every
kernel of one layer against its roofline.

    python bench.py --design piburax [--design-sizes 1b,8b]        (one JSON line)
    python benchmarks/bench_latent.py [--sizes 1b,8b] [--out FILE]

Random weights. Layer stacks are captured in a CUDA graph, so the times are device times; the weights of a stack
exceed L2 (126 MB). Single kernels are timed with an L2 flush (256 MB memset) before every launch. CUDA events, 5
warm-up runs, median. Roofline time = max(FLOPs / measured bf16 peak, bytes / measured copy bandwidth).
"""

from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np
import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

from benchmarks.bench_kernels import peaks, time_fn  # noqa: E402
from parallax_b200.cache.kv_pool import KVPool  # noqa: E402
from parallax_b200.engine.batch import BatchBuilder  # noqa: E402
from parallax_b200.models.config import config_from_hf, named_config  # noqa: E402
from parallax_b200.models.registry import build_stage  # noqa: E402
from parallax_b200.ops import cuda as cu  # noqa: E402

PAGE = 16
SLOTS = 128        # requests with a state of their own
LAYERS = {"1b": 12, "8b": 4}


def twin_of(cfg, layers: int):
    """DeepSeek-style dense decoder with the sizes of layer 0 of ``cfg``."""
    m, ff = cfg.layer_specs[0].mixer, cfg.layer_specs[0].mlp.ff
    return config_from_hf(dict(
        architectures=["DeepseekV3ForCausalLM"], model_type="deepseek_v3", hidden_size=cfg.hidden_size,
        num_hidden_layers=layers, num_attention_heads=m.heads, num_key_value_heads=m.heads, q_lora_rank=None,
        kv_lora_rank=m.kv_rank, qk_nope_head_dim=m.dim, qk_rope_head_dim=m.rot_dim, v_head_dim=m.vdim,
        intermediate_size=ff, vocab_size=1024, rope_theta=1e4, max_position_embeddings=16384))


def cut(cfg, layers: int, window=None):
    raw = dict(cfg.raw, vocab=1024, layers=cfg.raw["layers"][:1] * layers)
    if window is not None:
        e = json.loads(json.dumps(raw["layers"][0]))
        e["mixer"]["mask"]["size"] = window
        raw["layers"] = [e] * layers
    return config_from_hf(raw)


class Stack:
    """A stack of layers with its cache, and batches to run through it."""

    def __init__(self, cfg, tokens: int, device="cuda:0"):
        self.cfg, self.dev = cfg, torch.device(device)
        self.stage = build_stage(cfg, 0, cfg.num_hidden_layers, self.dev, torch.bfloat16, max_positions=16384)
        self.stage.init_random(1)
        self.blocks = -(-tokens // PAGE)
        self.pool = KVPool(cfg, 0, cfg.num_hidden_layers, self.blocks, PAGE, self.dev, torch.bfloat16,
                           num_linear_slots=SLOTS if cfg.has_linear_layers else 0)
        for lc in self.pool.layers:
            for t in (lc.k, lc.v, lc.conv_state, lc.rec_state):
                if t is not None:
                    t.normal_(0, 0.5)
        self.stage.attach_kv(self.pool.layers)

    def batch(self, prefill: list, decode: list):
        """``prefill``: prompt lengths, ``decode``: context lengths of decode rows."""
        pages = [-(-n // PAGE) for n in prefill + decode]
        assert sum(pages) <= self.blocks
        perm = np.random.default_rng(0).permutation(self.blocks).astype(np.int32)
        tables = np.zeros((len(pages), max(pages)), dtype=np.int32)
        o = 0
        for i, n in enumerate(pages):
            tables[i, :n] = perm[o:o + n]
            o += n
        pos = np.concatenate([np.arange(n) for n in prefill] + [np.asarray([n - 1 for n in decode])]).astype(np.int32) \
            if decode or prefill else np.zeros(0, np.int32)
        seq = np.concatenate([np.full(n, i) for i, n in enumerate(prefill)]
                             + [np.arange(len(prefill), len(pages))]).astype(np.int64)
        slots = tables[seq, pos // PAGE].astype(np.int64) * PAGE + pos % PAGE
        T, n_p = len(pos), len(prefill)
        b = BatchBuilder(self.dev, T, len(pages), tables.shape[1])
        fb = b.build(np.zeros(T, np.int32), pos, slots, prefill, prefill, tables[:n_p] if n_p else None,
                     np.asarray(decode, dtype=np.int32), tables[n_p:] if decode else None, np.zeros(0, np.int32),
                    np.arange(len(pages), dtype=np.int32))
        fb.keep = b
        return fb

    def time(self, fb, iters: int = 20) -> float:
        """Device ms of one pass of ``fb`` through the stack."""
        h = torch.randn(fb.num_tokens, self.cfg.hidden_size, device=self.dev).to(self.stage.hidden_dtype)
        with torch.inference_mode():
            s = torch.cuda.Stream()
            s.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(s):
                for _ in range(3):
                    self.stage.forward_layers(h.clone(), fb)
            torch.cuda.current_stream().wait_stream(s)
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, stream=s):      # (the GEMM's split-K scratch belongs to a stream)
                self.stage.forward_layers(h, fb)
            for _ in range(5):
                g.replay()
            ts = []
            for _ in range(iters):
                a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                a.record()
                g.replay()
                b.record()
                torch.cuda.synchronize()
                ts.append(a.elapsed_time(b))
        cu.check_status(self.dev)
        ts.sort()
        return ts[len(ts) // 2]


def keys_seen(n: int, window: int) -> int:
    """Sum over the positions of a prompt of ``n`` tokens of the keys each sees."""
    if not window or n <= window:
        return n * (n + 1) // 2
    return window * (window + 1) // 2 + (n - window) * window


def kernel_rows(stack: Stack, fb, label: str, keys: int, kv_tokens: int) -> list:
    """Every kernel of layer 0 on this batch: ms and roofline fraction. ``keys``: (query token, key) pairs;
    ``kv_tokens``: distinct cached rows read."""
    hbm, tf, _tag = peaks()
    st, cfg, T = stack.stage, stack.cfg, fb.num_tokens
    W, bf = cfg.hidden_size, torch.bfloat16
    rnd = lambda *s: (torch.randn(*s, device=stack.dev) * 0.3).to(bf)  # noqa: E731
    rows = []

    def add(name, fn, flops, byts):
        ms = time_fn(fn)
        roof = max(flops / (tf * 1e9), byts / (hbm * 1e6))
        rows.append(dict(batch=label, kernel=name, us=round(ms * 1e3, 1), roofline_frac=round(roof / ms, 3),
                         bound="compute" if flops / (tf * 1e9) > byts / (hbm * 1e6) else "memory"))

    def gemm(name, x, w, **kw):
        (M, K), N = x.shape, w.shape[0]
        n_out = N // 2 if kw.get("epi") in (cu.EPI_SILU_MUL, cu.EPI_CLIP_GLU) else N
        add(name, lambda: cu.linear(x, w, **kw), 2.0 * M * N * K, 2.0 * (M * K + N * K + M * n_out))

    x = rnd(T, W)
    lw = st.layers[0]
    cache = stack.pool.layers[0].k
    Tp = fb.num_prefill_tokens
    latent = hasattr(lw, "w_in")
    if latent:
        m = lw.spec.mixer
        H, L, R, V, dim, scale = m.heads, m.kv_rank, m.rot_dim, m.vdim, m.dim, m.scale
    else:
        H, L, R, V, dim, scale = st.H, st.L, st.R, st.V, st.nope, st.scale
    attn_flops, attn_bytes = 2.0 * keys * H * (2 * L + R), 2.0 * (kv_tokens * (L + R) + T * H * (2 * L + R))
    up_flops, uk_bytes, uv_bytes = 2.0 * T * H * L, 2.0 * (T * H * (dim + L) + H * L * dim), 2.0 * (T * H * (V + L) + H * L * V)
    if latent:
        gemm("q | latent | gate projection", x, lw.w_in)
        proj, q_cat = cu.linear(x, lw.w_in), torch.empty((T, H, L + R), dtype=bf, device=stack.dev)
        kv_off = H * m.q_width
        g_off = kv_off + m.row_width
        add("cache rows + query rotation", lambda: cu.latent_prep(
            proj, kv_off, H, m.q_width, dim, lw.kv_norm, lw.cos_sin, fb.positions, fb.slot_mapping, cache, q_cat, 1e-6, L, R,
            R), 0, 2.0 * T * (2 * (L + R) + 2 * H * R))
        add("key up-projection of q", lambda: cu.head_linear(proj, m.q_width, lw.w_uk_s, H, q_cat[:, :, :L]), up_flops * dim,
            uk_bytes)
        o_lat = torch.empty((T, H, L), dtype=bf, device=stack.dev)
        if Tp:
            add("attention", lambda: cu.latent_attn(q_cat, cache, fb.p_block_tables, fb.p_cu_q, fb.p_ctx_lens, scale, L,
                                                    m.window, lw.sinks, fb.p_max_q, fb.p_max_ctx, out=o_lat), attn_flops, attn_bytes)
        else:
            add("attention", lambda: cu.latent_attn(q_cat, cache, fb.d_block_tables, None, fb.d_ctx_lens, scale, L, m.window,
                                                    lw.sinks, 1, fb.d_max_ctx, out=o_lat), attn_flops, attn_bytes)
        heads = torch.empty((T, H, V), dtype=bf, device=stack.dev)
        gate = proj[:, g_off:g_off + H * V]
        add("value up-projection (+ gate)", lambda: cu.head_linear(o_lat.view(T, -1), L, lw.w_uv, H, heads, gate=gate),
            up_flops * V, uv_bytes + 2.0 * T * H * V)
        gemm("output projection", rnd(T, H * V), lw.w_o)
        h = torch.randn(T, W, device=stack.dev)
        add("residual + norm", lambda: cu.residual_norm(h, x, lw.norm1, 1e-6, 0.3), 0, T * W * 12.0)
        gemm("gate / up (+ clipped GLU)", x, lw.w_gu, epi=cu.EPI_CLIP_GLU, limit=6.0)
        gemm("down projection", rnd(T, lw.w_down.shape[1]), lw.w_down)
    else:
        gemm("q projection", x, lw.w_q_b)
        gemm("latent projection", x, lw.w_kv_a)
        kv, q = cu.linear(x, lw.w_kv_a), cu.linear(x, lw.w_q_b)
        add("cache rows", lambda: cu.mla_kv_prep(kv, lw.kv_a_norm, st.cos_sin, fb.positions, fb.slot_mapping, cache, 1e-6, L),
            0, 2.0 * T * 2 * (L + R))
        add("query rotation + key up-projection of q", lambda: cu.mla_q_absorb(q, lw.w_uk_s, st.cos_sin, fb.positions, H, dim, L),
            up_flops * dim, uk_bytes)
        q_lat, q_pe = cu.mla_q_absorb(q, lw.w_uk_s, st.cos_sin, fb.positions, H, dim, L)
        o_lat = torch.empty_like(q_lat)
        bt, cq = (fb.p_block_tables, fb.p_cu_q) if Tp else (fb.d_block_tables, None)
        add("attention", lambda: cu.mla_attn(q_lat, q_pe, cache, bt, cq, fb.positions, scale, 0, T, out=o_lat), attn_flops,
            attn_bytes)
        add("value up-projection", lambda: cu.mla_unabsorb(o_lat, lw.w_uv_s, T), up_flops * V, uv_bytes)
        gemm("output projection (+ residual)", rnd(T, H * V), lw.w_o, residual=x)
        add("norm", lambda: cu.rmsnorm(x, lw.ln1, 1e-6), 0, T * W * 4.0)
        gemm("gate / up (+ SwiGLU)", x, lw.w_gu, epi=cu.EPI_SILU_MUL)
        gemm("down projection (+ residual)", rnd(T, lw.w_down.shape[1]), lw.w_down, residual=x)
    cu.check_status(stack.dev)
    return rows


def run(sizes: list, log=print) -> dict:
    table, kernels = [], []
    for size in sizes:
        base, n = named_config(f"piburax-{size}"), LAYERS[size]
        window = base.layer_specs[0].mixer.window
        models = [("piburax", cut(base, n), window), ("piburax, no window", cut(base, n, 0), 0), ("mla twin", twin_of(base, n), 0)]
        for name, cfg, win in models:
            st = Stack(cfg, 264 * 2048)
            for label, prefill, decode in ((f"prefill 1 x {window}", [window], []), ("prefill 1 x 4096", [4096], []),
                                           ("prefill 8 x 512", [512] * 8, []), (f"decode 1 x {window}", [], [window]),
                                           (f"decode 32 x {window}", [], [window] * 32), ("decode 128 x 2048", [], [2048] * 128)):
                fb = st.batch(prefill, decode)
                ms = st.time(fb)
                row = dict(size=size, model=name, batch=label, layers=n, ms_per_layer=round(ms / n, 4),
                           tokens_per_s_per_layer=round(fb.num_tokens / (ms / n) * 1e3))
                table.append(row)
                log(row)
                if (size == "8b" or len(sizes) == 1) and name != "piburax, no window" and \
                        label in ("prefill 1 x 4096", f"decode 32 x {window}", "decode 128 x 2048"):
                    keys = sum(keys_seen(p, win) for p in prefill) + sum(min(c, win) if win else c for c in decode)
                    kv = sum(prefill) + sum(min(c, win) if win else c for c in decode)
                    for r in kernel_rows(st, fb, label, keys, kv):
                        kernels.append(dict(size=size, model=name, **r))
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
