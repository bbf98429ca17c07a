"""Every mechanism of the Zudepel layers alone: the op (CPU restatement or B200 kernel) against the equations in
``helpers/zudepel_oracle.py``, with inputs that make a single wrong key, tap, decay, sink or expert stand out."""

import math

import pytest
import torch

from helpers import zudepel_oracle as oracle
from parallax_b200 import ops

GPU = pytest.mark.gpu
TARGETS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda:0", torch.float32), id="gpu-fp32", marks=GPU),
           pytest.param(("cuda:0", torch.bfloat16), id="gpu-bf16", marks=GPU)]


def gen(seed=0):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g)


def rel(got, want):
    got, want = got.double().cpu(), want.double()
    return float((got - want).norm() / want.norm())


def tol(dt, f32=3e-6, bf16=6e-3):
    return f32 if dt == torch.float32 else bf16


def status_ok(dev):
    if dev != "cpu":
        from parallax_b200.ops import cuda as cu

        cu.check_status(torch.device(dev))


def i32(x, dev):
    return torch.tensor(x, dtype=torch.int32, device=dev)


class Steps:
    """Sequences cut into steps of one batch each, slices first and decoded tokens behind them, the way the engine lays
    them out: yields (rows of the concatenated sequences, positions, seq_cu, slots, slices, tokens in slices, starts)."""

    def __init__(self, lens, plan, dev):
        self.lens, self.plan, self.dev = lens, plan, dev

    def __iter__(self):
        at, base = [0] * len(self.lens), [sum(self.lens[:i]) for i in range(len(self.lens))]
        k = 0
        while any(a < n for a, n in zip(at, self.lens)):
            counts = self.plan[k % len(self.plan)]
            k += 1
            todo = [(s, min(c, self.lens[s] - at[s])) for s, c in enumerate(counts) if min(c, self.lens[s] - at[s]) > 0]
            slices = [(s, c) for s, c in todo if c > 1 or at[s] == 0]
            order = slices + [(s, c) for s, c in todo if not (c > 1 or at[s] == 0)]
            rows, pos, cu = [], [], [0]
            for s, c in order:
                rows += range(base[s] + at[s], base[s] + at[s] + c)
                pos += range(at[s], at[s] + c)
                cu.append(cu[-1] + c)
                at[s] += c
            yield (torch.tensor(rows, dtype=torch.long), i32(pos, self.dev), i32(cu, self.dev), [s for s, _ in order],
                   len(slices), sum(c for _, c in slices))


PLANS = {"whole": [(999, 999, 999)], "tokens": [(1, 1, 1)], "mixed": [(5, 1, 70), (1, 2, 1), (64, 1, 3), (2, 9, 1), (1, 1, 65)]}


# ---------------------------------------------------------------------------------- convolution, norms, rotation, cache
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("plan", sorted(PLANS))
@pytest.mark.parametrize("H,G,dk,dv,rot,taps", [(3, 1, 7, 5, 6, 3), (4, 2, 24, 16, 16, 4), (2, 2, 64, 72, 64, 1), (4, 4, 16, 16, 16, 2),
                                                (3, 0, 16, 8, 16, 5), (2, 1, 40, 24, 8, 0)])
def test_convolution_norm_rotation_and_cache_rows(target, plan, H, G, dk, dv, rot, taps):
    """Slices of any size beside decoded tokens; state slots and pages start out dirty; zeros behind padded heads."""
    dev, dt = target
    rnd = gen(H * dk + taps)
    lens, eps, base, page = [40, 3, 90], 1e-5, 500.0, 16
    widths = [H * dk, G * dk, G * dv]
    offs = (8, 8 + widths[0] + 8 - widths[0] % 8, 0)
    offs = (offs[0], offs[1], offs[1] + widths[1] + 8 - widths[1] % 8)
    u = rnd(sum(lens), offs[2] + widths[2] + 8).to(dt)
    C, cols = sum(widths), max(dk, dv) + 8
    conv = rnd(C, taps).to(dt) if taps else None
    qn, kn = 1 + 0.3 * rnd(H * dk), 1 + 0.3 * rnd(max(G * dk, 1))
    state = torch.full((5, max(taps - 1, 0), C), 30.0, dtype=dt, device=dev)
    tables = torch.randperm(20, generator=torch.Generator().manual_seed(1))[:18].view(3, 6)
    kc, vc = (torch.full((20, G, page, cols), 9.0, dtype=dt, device=dev) for _ in range(2)) if G else (None, None)
    cos_sin = ops.build_cos_sin(128, rot, base, device=dev)
    q_all = torch.zeros(sum(lens), H, cols)
    seq_of = torch.repeat_interleave(torch.arange(3), torch.tensor(lens))
    for rows, pos, cu, seqs, slices, slice_tokens in Steps(lens, PLANS[plan], dev):
        p = pos.cpu().long()
        slot = tables[seq_of[rows], p // page] * page + p % page
        q = torch.full((len(rows), H, cols), 7.0, dtype=dt, device=dev)
        ops.conv_qkv_prep(u[rows].to(dev), offs, H, G, dk, dv, None if conv is None else conv.t().contiguous().to(dev), state,
                          qn.to(dev), kn.to(dev), cos_sin, pos, cu, i32([4 - s for s in seqs], dev), slices, slice_tokens,
                          slot.to(dev), kc, vc, q, eps)
        q_all[rows] = q.float().cpu()
    status_ok(dev)
    for s in range(3):
        lo, hi = sum(lens[:s]), sum(lens[:s + 1])
        parts = [u[lo:hi, o:o + n].double() for o, n in zip(offs, widths)]
        if taps:
            parts = [oracle.causal_conv(x, c) for x, c in zip(parts, conv.split(widths))]
        slots = (tables[s][torch.arange(hi - lo) // page] * page + torch.arange(hi - lo) % page)
        want_q = oracle.split_heads(oracle.rms_norm(parts[0], qn, eps), H, dk)
        for h in range(H):
            assert rel(q_all[lo:hi, h, :dk], oracle.rotate_half(want_q[h], base, rot)) < tol(dt, 5e-6)
        assert bool((q_all[lo:hi, :, dk:] == 0).all())
        for g in range(G):
            k = oracle.rotate_half(oracle.split_heads(oracle.rms_norm(parts[1], kn, eps), G, dk)[g], base, rot)
            got_k, got_v = (c.transpose(1, 2).reshape(-1, G, cols)[slots.to(dev), g].cpu() for c in (kc, vc))
            assert rel(got_k[:, :dk], k) < tol(dt, 5e-6) and rel(got_v[:, :dv], parts[2][:, g * dv:(g + 1) * dv]) < tol(dt)
            assert bool((got_k[:, dk:] == 0).all()) and bool((got_v[:, dv:] == 0).all())


# ---------------------------------------------------------------------------------- lightning attention
def lightning_case(target, H, dk, dv, decay, u, lens, plan, fill=50.0):
    dev, dt = target
    offs = (0, H * dk + -(H * dk) % 8, 2 * (H * dk + -(H * dk) % 8))
    pw = (torch.tensor(decay, dtype=torch.float64)[:, None] ** torch.arange(65)).float().to(dev)
    state = torch.full((4, H, dk, dv), fill, device=dev)
    out = torch.zeros(sum(lens), H, dv)
    for rows, pos, cu, seqs, slices, _n in Steps(lens, plan, dev):
        got = ops.lightning_attn(u[rows].to(dev), offs, H, dk, dv, pw, state, pos, cu, i32([3 - s for s in seqs], dev), slices)
        out[rows] = got.float().cpu()
    status_ok(dev)
    return out, state, offs


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,dk,dv", [(3, 16, 8), (2, 64, 40), (2, 128, 128), (3, 9, 7), (2, 96, 33), (1, 200, 64), (1, 264, 12)])
def test_lightning_attention(target, H, dk, dv):
    """Prompts, slices and single tokens over chunk edges, decays from 0 to 1, against the explicit sum; the state after a
    prompt is the state after its tokens one by one."""
    dev, dt = target
    lens, rnd = [150, 65, 200], gen(dk)
    width = 2 * (H * dk + -(H * dk) % 8) + H * dv
    u = (1.5 * rnd(sum(lens), width + -width % 8)).to(dt)
    decay = [(0.97, 1.0, 0.0)[h % 3] for h in range(H)]
    results, want = {}, {}
    for name, plan in PLANS.items():
        got, results[name], offs = lightning_case(target, H, dk, dv, decay, u, lens, plan)
        for s in range(3):
            lo, hi = sum(lens[:s]), sum(lens[:s + 1])
            q, k, v = (oracle.silu(u[lo:hi, o:o + H * d].double()).to(dt).double() for o, d in zip(offs, (dk, dk, dv)))
            for h in range(H):
                if (s, h) not in want:
                    want[s, h] = oracle.decayed_sum(q[:, h * dk:(h + 1) * dk], k[:, h * dk:(h + 1) * dk],
                                                    v[:, h * dv:(h + 1) * dv], decay[h])
                assert rel(got[lo:hi, h], want[s, h]) < tol(dt, 1e-5, 4e-3), (name, s, h)
    assert bool((results["whole"][0] == 50).all())       # the slot nobody holds
    for name in ("whole", "mixed"):
        # products of fp32 operands go through two bf16 numbers each: far better than one bf16 rounding
        assert rel(results[name][1:], results["tokens"][1:].cpu()) < 2e-5, name


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("dk,dv", [(16, 8), (128, 128)])
def test_one_far_key_is_still_there(target, dk, dv):
    """A large key and value at one place, small ones elsewhere: what a later token reads of it is decay^distance, right
    before and after the chunk edges, in prompts and in decoding."""
    dev, dt = target
    n, decay, rnd = 200, 0.98, gen(3)
    off = dk + -dk % 8
    for at in (0, 1, 62, 63, 64, 65, 127, 128, 198):
        u = (0.01 * rnd(n, 2 * off + dv + -dv % 8)).to(dt)
        u[:, 0] = 8.0
        u[at, off] = 20.0
        u[at, 2 * off:2 * off + dv] = 10.0
        for plan in ([(n,)], [(at + 1,), (1,)], [(63,), (2,)]):
            got, _state, _offs = lightning_case(target, 1, dk, dv, [decay], u, [n], plan)
            want = 8.0 * 20.0 * 10.0 * decay ** torch.arange(n - at, dtype=torch.float64)
            assert float((got[at:, 0, 0].double() / want - 1).abs().max()) < 1e-2, (at, plan)
            assert float(got[:at].abs().max() if at else 0.0) < 1.0


# ---------------------------------------------------------------------------------- gates
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,dv,cols,pad", [(3, 5, 8, 1), (4, 16, 64, 0), (8, 128, 128, 0), (40, 72, 128, 0)])
@pytest.mark.parametrize("normed", [False, True])
def test_gated_heads(target, heads, dv, cols, pad, normed):
    dev, dt = target
    rnd = gen(dv)
    N = heads * dv
    x, g, w = rnd(6, heads, cols).to(dt), (2 * rnd(6, N + 8)).to(dt), 1 + 0.3 * rnd(N)
    x[3] *= 1e-3                      # eps matters
    buf = torch.full((6, N + pad + 8), float("nan"), dtype=dt, device=dev)
    gate = g.to(dev)[:, :N]
    ops.gated_rows(x.to(dev), dv, gate, buf[:, :N + pad], w.to(dev) if normed else None, 1e-5)
    want = x[:, :, :dv].reshape(6, N).double()
    if normed:
        want = oracle.rms_norm(want, w, 1e-5)
    assert rel(buf[:, :N], want * oracle.sigmoid(g[:, :N].double())) < tol(dt)
    assert bool((buf[:, N:N + pad] == 0).all()) and bool(buf[:, N + pad:].isnan().all())


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("rows,width,ff", [(3, 30, 64), (70, 128, 192), (300, 256, 512)])
def test_gated_linear_units(target, rows, width, ff):
    dev, dt = target
    rnd = gen(ff)
    x, gate, up = (2 * rnd(rows, width)).to(dt), (rnd(ff, width) / width ** 0.5).to(dt), (rnd(ff, width) / width ** 0.5).to(dt)
    w = ops.interleave_gate_up(gate, up).to(dev)
    scale = torch.randn(rows, 3, generator=torch.Generator().manual_seed(1)).to(dev)
    for act, fn in ((0, oracle.silu), (2, oracle.gelu_tanh)):
        want = fn(x.double() @ gate.double().T) * (x.double() @ up.double().T)
        assert rel(ops.glu_linear(x.to(dev), w, act), want) < tol(dt, 3e-6, 5e-3)
        buf = torch.full((rows, ff + 16), 3.0, dtype=dt, device=dev)
        ops.glu_linear(x.to(dev), w, act, scale[:, 1], buf[:, 8:8 + ff])
        assert rel(buf[:, 8:8 + ff], want * oracle.sigmoid(scale[:, 1:2].double().cpu())) < tol(dt, 3e-6, 5e-3)
        assert bool((buf[:, :8] == 3).all()) and bool((buf[:, 8 + ff:] == 3).all())
    status_ok(dev)


def test_gelu_far_from_zero():
    z = torch.tensor([-80.0, -12.0, -3.0, -1e-4, 0.0, 1e-4, 3.0, 12.0, 80.0], dtype=torch.float32)
    want = oracle.gelu_tanh(z.double())
    got = ops.glu_linear(z[:, None], ops.interleave_gate_up(torch.eye(64)[:, :1].contiguous(), torch.ones(64, 1)), 2)[:, 0] / z
    ok = z != 0
    assert float((got.double() - want)[ok].abs().max()) < 1e-6


@GPU
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_gelu_far_from_zero_on_the_gpu(dt):
    z = torch.tensor([-80.0, -12.0, -3.0, -0.01, 0.01, 3.0, 12.0, 80.0])
    x = torch.zeros(8, 64)
    x[:, 0], x[:, 1] = z, 1.0
    gate, up = torch.zeros(64, 64), torch.zeros(64, 64)
    gate[0, 0] = up[0, 1] = 1.0
    got = ops.glu_linear(x.to("cuda:0", dt), ops.interleave_gate_up(gate, up).to("cuda:0", dt), 2)[:, 0]
    want = oracle.gelu_tanh(x[:, 0].to(dt).double())
    assert float((got.cpu().double() - want).abs().max()) < (2e-6 if dt == torch.float32 else 0.3)
    assert not bool(got.isnan().any()) and float(got[:2].abs().max()) < 1e-6


# ---------------------------------------------------------------------------------- router and experts
@pytest.mark.parametrize("target", TARGETS[:2])
@pytest.mark.parametrize("E,top,groups", [(6, 2, None), (8, 3, (4, 2)), (8, 2, (2, 1)), (140, 9, (20, 3)), (512, 16, None), (9, 9, None), (12, 1, (12, 5))])
def test_routing(target, E, top, groups):
    """Corrections large enough to overrule the scores and to make every choice score negative; weights without them; logits
    in wider rows."""
    dev, _ = target
    rnd = gen(E)
    z, corr = 2 * rnd(50, E + 5), 0.3 * rnd(E) - 1.5
    ids, w = ops.moe_route(z.to(dev)[:, 2:2 + E], corr.to(dev), top, 0, True, *(groups or (1, 1)), group_top=1)
    for t in range(50):
        s = oracle.router_scores(z[t, 2:2 + E].double())
        want = oracle.choose(s, corr.double(), top, groups and {"count": groups[0], "keep": groups[1]})
        assert ids[t].tolist() == want
        ws = s[want] / (s[want].sum() + 1e-20)
        assert float((w[t].double().cpu() - ws).abs().max()) < 2e-6
    sig, _w = ops.moe_route(z.to(dev)[:, 2:2 + E], None, top, 1)          # the sigmoid mode still routes by score
    assert sorted(sig[0].tolist()) == sorted(z[0, 2:2 + E].topk(top).indices.tolist())


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("rows,W,ff,experts,identity,top,groups,shared",
                         [(3, 30, 24, 4, 2, 2, None, 40), (40, 128, 64, 6, 0, 2, (2, 1), None), (1, 320, 100, 5, 3, 3, (4, 3), 64),
                          (200, 200, 72, 12, 4, 4, (4, 2), 96), (5, 64, 64, 2, 6, 3, None, 64)])
def test_routed_feed_forward(target, rows, W, ff, experts, identity, top, groups, shared):
    """Experts that nobody chooses, identity experts, padded sizes; the update of the residual and the next norm."""
    from parallax_b200.models.layer_spec import parse_layers
    from parallax_b200.models.moe import RoutedExperts

    dev, dt = target
    mlp = oracle.moe(ff=ff, experts=experts, top=top, identity=identity, groups=groups, shared=shared)
    cfg = oracle.random_config([oracle.lightning(mlp=mlp)], width=W)
    w = oracle.random_weights(cfg, seed=W)
    spec = parse_layers("Zudepel", cfg["layers"])[0].mlp
    moe = RoutedExperts.build(spec, lambda n, d=dt: w["l0.mlp." + n].to(dev, d), dev)
    rnd = gen(W)
    h, x, y, nw = rnd(rows, W).to(dt), rnd(rows, W), rnd(rows, W + 8)[:, :W].to(dt), 1 + 0.2 * rnd(W)
    chosen = []
    want = oracle.routed(dict(mlp, shared=None), w, "l0.mlp.", h.double(), chosen)
    xg = x.to(dev).clone()
    routed, gate = moe.forward(h.to(dev))
    low = ops.residual_add(xg, y.to(dev), nw.to(dev), 1e-5, routed, h.to(dev))
    status_ok(dev)
    total = x.double() + y.double() + want
    assert rel(xg - x.to(dev) - y.to(dev).float(), want) < tol(dt, 1e-5, 8e-3)
    assert low.dtype == dt and rel(low, oracle.rms_norm(total, nw, 1e-5)) < tol(dt, 1e-5, 8e-3)
    if shared:
        assert rel(gate, (h.double() @ w["l0.mlp.shared.sg"].double().T)[:, 0]) < tol(dt, 1e-5, 1e-2)
    if identity:
        assert any(e >= experts for ids in chosen for e in ids) and any(e < experts for ids in chosen for e in ids)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("width", [30, 64, 320, 4096, 20000])
def test_residual_add(target, width):
    dev, dt = target
    rnd = gen(width)
    x, y, w = rnd(4, width), (3 * rnd(4, width)).to(dt), 1 + 0.3 * rnd(width)
    x[2], y[2] = 1e-4 * x[2], 0 * y[2]
    xg = x.to(dev).clone()
    low = ops.residual_add(xg, y.to(dev), w.to(dev), 1e-6)
    want = x.double() + y.double()
    assert rel(xg, want) < 1e-6 and low.dtype == dt and rel(low, oracle.rms_norm(want, w, 1e-6)) < tol(dt, 3e-6, 4e-3)
    assert ops.residual_add(xg, y.to(dev)) is None and rel(xg, want + y.double()) < 1e-6


# ---------------------------------------------------------------------------------- attention over pages
class Paged:
    """Keys and values on shuffled pages, with helpers to run and to restate attention."""

    def __init__(self, target, H, G, D, page, ctxs, seed=0, scale_k=0.5):
        self.dev, self.dt = target
        self.H, self.G, self.D, self.page, self.ctxs = H, G, D, page, ctxs
        self.rnd = gen(seed)
        pages = [-(-c // page) for c in ctxs]
        perm = torch.randperm(sum(pages) + 3, generator=torch.Generator().manual_seed(seed))
        self.tables, o = torch.zeros(len(ctxs), max(pages), dtype=torch.int32), 0
        for i, k in enumerate(pages):
            self.tables[i, :k] = perm[o:o + k].int()
            o += k
        shape = (sum(pages) + 3, G, page, D)
        self.k, self.v = (scale_k * self.rnd(*shape)).to(self.dt), self.rnd(*shape).to(self.dt)
        self.scale = 1.3 * D ** -0.5

    def at(self, cache, b, pos):
        return cache[int(self.tables[b, pos // self.page]), :, pos % self.page]      # [G, D], a view

    def run(self, q, q_lens, sinks, decode):
        d = lambda t: t.to(self.dev)  # noqa: E731
        ctx = i32(self.ctxs, self.dev)
        args = (d(q), d(self.k), d(self.v), d(self.tables))
        if decode:
            out = ops.attn_decode(*args, ctx, self.scale, sinks=d(sinks), max_ctx=max(self.ctxs))
        else:
            cu = i32([0] + torch.tensor(q_lens).cumsum(0).tolist(), self.dev)
            out = ops.attn_prefill(*args, cu, ctx, max(q_lens), self.scale, sinks=d(sinks))
        status_ok(self.dev)
        return out

    def want(self, q, q_lens, sinks):
        out, t = torch.zeros(q.shape, dtype=torch.float64), 0
        for b, n in enumerate(q_lens):
            ctx = self.ctxs[b]
            for h in range(self.H):
                k, v = (torch.stack([self.at(c, b, i)[h // (self.H // self.G)] for i in range(ctx)]).double() for c in (self.k, self.v))
                full = torch.zeros(ctx, self.D, dtype=torch.float64)
                full[ctx - n:] = q[t:t + n, h].double()
                out[t:t + n, h] = oracle.attend(full, k, v, self.scale, sinks[h])[ctx - n:]
            t += n
        return out


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,G,D,page", [(3, 3, 24, 16), (6, 2, 64, 16), (8, 8, 128, 16), (40, 2, 64, 16), (4, 1, 200, 32), (8, 2, 128, 64)])
def test_attention_of_ragged_batches(target, H, G, D, page):
    for q_lens, ctxs, decode in (([1, 1, 1, 1], [1, 16, 34, 150], True), ([9, 2, 1], [9, 67, 40], False), ([130], [140], False)):
        pg = Paged(target, H, G, D, page, ctxs, seed=H)
        q = pg.rnd(sum(q_lens), H, D).to(pg.dt)
        sinks = 2 * pg.rnd(H)
        assert rel(pg.run(q, q_lens, sinks, decode), pg.want(q, q_lens, sinks)) < tol(pg.dt, 3e-6, 8e-3)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,G,D", [(2, 2, 24), (4, 2, 64), (4, 1, 128)])
def test_one_key_stands_out(target, H, G, D):
    """One key matches the query so well that it takes the whole softmax wherever it is: the first tokens, page and tile
    borders, the token itself; a query before it must not see it. Large and very negative sinks do and do not take it."""
    ctx, n = 180, 60
    for at in (0, 1, 15, 16, 63, 64, 127, 128, ctx - n, ctx - 2, ctx - 1):
        pg = Paged(target, H, G, D, 16, [ctx], seed=at, scale_k=0.02)
        dirs = pg.rnd(D)
        dirs = dirs / dirs.norm()
        pg.at(pg.k, 0, at)[:] = (dirs * 30).to(pg.dt)
        pg.at(pg.v, 0, at)[:] = 100.0
        q = (dirs * 30).to(pg.dt).expand(n, H, D).contiguous()
        sinks = torch.full((H,), -50.0)
        sinks[0] = 30.0 * 30.0 * pg.scale + 3
        got, want = pg.run(q, [n], sinks, False), pg.want(q, [n], sinks)
        one = pg.run(q[:1], [1], sinks, True)
        assert rel(one, want[-1:]) < 2e-2
        for i in range(n):
            seen = at <= ctx - n + i
            assert (float(got[i, 1].float().mean()) > 90) == seen, (at, i)
            assert float((got[i].double().cpu() - want[i]).abs().max()) < 1.0
        assert float(got[-1, 0].float().mean()) < 10       # the sink of head 0 outweighs the key


@pytest.mark.parametrize("target", TARGETS)
def test_rows_do_not_depend_on_their_neighbours(target):
    """A query's result is the same bits alone and in a batch, and on other pages."""
    pg = Paged(target, 4, 2, 24, 16, [70, 200, 33], seed=5)
    q, sinks = pg.rnd(3, 4, 24).to(pg.dt), pg.rnd(4)
    whole = pg.run(q, [1, 1, 1], sinks, True)
    for b in range(3):
        alone = Paged(target, 4, 2, 24, 16, [pg.ctxs[b]], seed=99)
        for i in range(pg.ctxs[b]):
            for c, src in ((alone.k, pg.k), (alone.v, pg.v)):
                alone.at(c, 0, i).copy_(pg.at(src, b, i))
        assert torch.equal(alone.run(q[b:b + 1], [1], sinks, True)[0], whole[b])


# ---------------------------------------------------------------------------------- errors are reported, not followed
@GPU
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_indices_outside_the_pools_are_reported(dt):
    from parallax_b200.ops import KernelError

    target = ("cuda:0", dt)
    u = torch.zeros(4, 56).to(dt)
    with pytest.raises(KernelError, match="index"):
        ops_slots = lambda seqs: i32([77] * len(seqs), "cuda:0")  # noqa: E731
        pw = torch.ones(1, 65, device="cuda:0")
        ops.lightning_attn(u.cuda(), (0, 16, 32), 1, 16, 24, pw, torch.zeros(2, 1, 16, 24, device="cuda:0"), i32(range(4), "cuda:0"),
                           i32([0, 4], "cuda:0"), ops_slots([0]), 1)
        status_ok("cuda:0")
    pg = Paged(target, 2, 2, 24, 16, [40])
    pg.tables[0, 1] = 10 ** 6
    with pytest.raises(KernelError, match="block"):
        pg.run(pg.rnd(1, 2, 24).to(dt), [1], torch.zeros(2), True)
    assert math.isfinite(float(pg.k.float().sum()))
