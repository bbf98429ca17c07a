"""Every mechanism of the Zasalix layers alone: the op (CPU restatement or B200 kernel) against the equations in
``helpers/zasalix_oracle.py``, with inputs that make a single wrong key, window edge, gate or expert stand out."""

import math

import pytest
import torch

from helpers import zasalix_oracle as oracle
from parallax_b200 import ops
from parallax_b200.models.layer_spec import MEMORY_SLICE, memory_words

GPU = pytest.mark.gpu
TARGETS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda:0", torch.float32), id="gpu-fp32", marks=GPU),
           pytest.param(("cuda:0", torch.bfloat16), id="gpu-bf16", marks=GPU)]


def gen(seed=0):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g)


def rel(got, want):
    got, want = got.double().cpu(), want.double()
    return float((got - want).norm() / want.norm())


def tol(dt, f32=2e-6, bf16=6e-3):
    return f32 if dt == torch.float32 else bf16


def status_ok(dev):
    if dev != "cpu":
        from parallax_b200.ops import cuda as cu

        cu.check_status(torch.device(dev))


def i32(x, dev):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def steps(lens, plan):
    """Sequences cut into steps of one batch each, slices first and decoded tokens behind them, as the engine lays them out:
    (rows of the concatenated sequences, positions, ranges, sequences, number of slices, tokens in slices)."""
    at, base, k = [0] * len(lens), [sum(lens[:i]) for i in range(len(lens))], 0
    while any(a < n for a, n in zip(at, lens)):
        counts, k = plan[k % len(plan)], k + 1
        todo = [(s, min(c, lens[s] - at[s])) for s, c in enumerate(counts) if min(c, lens[s] - at[s]) > 0]
        slices = [(s, c) for s, c in todo if c > 1 or at[s] == 0]
        rows, pos, cu, order = [], [], [0], slices + [x for x in todo if x not in slices]
        for s, c in order:
            rows += range(base[s] + at[s], base[s] + at[s] + c)
            pos += range(at[s], at[s] + c)
            cu.append(cu[-1] + c)
            at[s] += c
        if order:
            yield torch.tensor(rows), pos, cu, [s for s, _ in order], len(slices), sum(c for _, c in slices)


PLANS = {"whole": [(999, 999, 999)], "tokens": [(1, 1, 1)], "mixed": [(5, 1, 70), (1, 2, 1), (64, 1, 3), (2, 9, 1), (1, 1, 65)]}


# ---------------------------------------------------------------------------------- tanh norms and the residual
def norm_weights(rnd, W, alpha):
    return 1 + 0.3 * rnd(W), 0.2 * rnd(W), alpha


def on(n, dev):
    return n[0].to(dev), n[1].to(dev), n[2]


def want_norm(x, n):
    return oracle.tanh_norm(x.double(), {"n": n[0], "n.b": n[1], "n.alpha": torch.tensor(n[2], dtype=torch.float64)}, "n")


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("W", [7, 48, 200, 3000, 4096])
def test_tanh_norm(target, W):
    """From deep in the linear range to saturation, rows picked and not."""
    dev, dt = target
    rnd = gen(W)
    x = rnd(9, W) * torch.tensor([1e-4, 1e-2, 0.3, 1, 1, 3, 10, 1e3, 0]).view(9, 1)
    n = norm_weights(rnd, W, 0.8)
    n[1][:] = 0 if W == 48 else n[1]
    got = ops.tanh_norm(x.to(dev), *on(n, dev), dtype=dt)
    assert got.dtype == dt
    for t in range(9 if W != 48 else 8):
        assert rel(got[t:t + 1], want_norm(x[t:t + 1], n)) < tol(dt, 5e-7, 3e-3), t
    rows = [4, 0, 8, 4]
    got = ops.tanh_norm(x.to(dev), *on(n, dev), rows=i32(rows, dev), dtype=dt)
    assert rel(got, want_norm(x[rows], n)) < tol(dt, 5e-7, 3e-3)
    status_ok(dev)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("W", [5, 64, 264, 2048, 4096 + 8, 9000])
@pytest.mark.parametrize("post", ["tanh", "rms", None])
@pytest.mark.parametrize("extra", ["none", "experts", "shared+experts", "entry"])
def test_residual_step(target, W, post, extra):
    dev, dt = target
    rnd, T, eps, k = gen(W), 6, 1e-3, 3
    x0, y = 2 * rnd(T, W), 0.7 * rnd(T, W).to(dt)
    n_post, n_pre, rms_w = norm_weights(rnd, W, 0.9), norm_weights(rnd, W, 0.4), 1 + 0.2 * rnd(W)
    rows, pos = rnd(40, W + -W % 64).to(dt), torch.randperm(40)[:T * k].view(T, k)
    table, ids, step = rnd(11, W).to(dt), [3, 0, 10, 3, 7, 1], 0.5 * rnd(W)
    if post is None and "experts" in extra:
        return
    want, kw = x0.double(), {}
    if post is not None:
        z = torch.zeros(T, W, dtype=torch.float64) if extra == "experts" else y.double()
        if "experts" in extra:
            z = z + sum(rows.double()[pos[:, j], :W] for j in range(k))
            kw["routed"] = (rows.to(dev), pos.to(torch.int32).to(dev), None)
        want = want + (want_norm(z, n_post) if post == "tanh" else oracle.over_rms(z, eps) * rms_w.double())
        kw.update(y=None if extra == "experts" else y.to(dev), post=on(n_post, dev) if post == "tanh" else (rms_w.to(dev),))
    if extra == "entry":
        want = want + table.double()[ids] + step.double()
        kw.update(table=table.to(dev), ids=i32(ids, dev), step=step.to(dev))
    for pre in (None, (), n_pre):
        x = x0.clone().to(dev)
        got = ops.residual_step(x, pre=pre and on(pre, dev), dtype=dt, eps=eps, **kw)
        status_ok(dev)
        assert rel(x, want) < 1e-6
        assert (got is None) if pre is None else rel(got, want_norm(want, n_pre) if pre else want) < tol(dt, 2e-6, 4e-3)


# ---------------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,d,R,L,rank,rot", [(3, 5, 6, 9, 11, 6), (4, 16, 8, 40, 24, 4), (2, 64, 32, 96, 64, 32)])
def test_latent_rows_and_queries(target, H, d, R, L, rank, rot):
    dev, dt = target
    rnd, T, eps, base, page = gen(H + L), 21, 1e-2, 300.0, 16
    q_off, kv_off = 8, 8 + rank + -rank % 8
    proj = rnd(T, kv_off + L + R + 5).to(dt)
    qn, kn = 1 + 0.3 * rnd(rank), 1 + 0.3 * rnd(L)
    pos = torch.arange(T) + 40
    slots = torch.randperm(5 * page)[:T]
    slots[3] = -1
    cache = torch.full((5, 1, page, L + R), 9.0, dtype=dt, device=dev)
    cos_sin = ops.build_cos_sin(128, rot, base, device=dev)
    c_q = torch.empty(T, rank, dtype=dt, device=dev)
    ops.latent_rows(proj.to(dev), q_off, qn.to(dev), c_q, kv_off, kn.to(dev), cos_sin, i32(pos.tolist(), dev), slots.to(dev),
                    cache, eps, L, R, rot)
    q = rnd(T, H * (d + R) + 3).to(dt)
    q_cat = torch.full((T, H, L + R), 7.0, dtype=dt, device=dev)
    ops.latent_queries(q.to(dev), H, d + R, d, cos_sin, i32(pos.tolist(), dev), q_cat, L, R, rot)
    status_ok(dev)
    assert rel(c_q, oracle.over_rms(proj[:, q_off:q_off + rank].double(), eps) * qn.double()) < tol(dt)

    def at_40(x):     # rows at positions 40 ..
        return oracle.rotate_neighbours(torch.cat([torch.zeros(40, x.shape[1], dtype=torch.float64), x.double()]), base, rot)[40:]

    want = torch.cat([oracle.over_rms(proj[:, kv_off:kv_off + L].double(), eps) * kn.double(),
                      at_40(proj[:, kv_off + L:kv_off + L + R])], -1)
    ok = slots >= 0
    assert rel(cache.view(-1, L + R).cpu()[slots[ok]], want[ok]) < tol(dt)
    other = torch.ones(5 * page, dtype=torch.bool)
    other[slots[ok]] = False
    assert bool((cache.view(-1, L + R).cpu()[other] == 9).all())
    for h in range(H):
        assert rel(q_cat[:, h, L:], at_40(q[:, h * (d + R) + d:(h + 1) * (d + R)])) < tol(dt)
    assert bool((q_cat[:, :, :L] == 7).all())


# ---------------------------------------------------------------------------------- windowed attention
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,G,dk,dv,rot", [(3, 1, 7, 5, 6), (4, 2, 24, 16, 8), (2, 2, 64, 72, 64), (4, 1, 40, 56, 16)])
def test_rotation_and_cache_rows(target, H, G, dk, dv, rot):
    """No convolution, no norms: rotated queries and keys, plain values, zeros behind padded heads, other rows untouched."""
    dev, dt = target
    rnd, T, base, page, first = gen(H * dk), 37, 500.0, 16, 50
    widths = [H * dk, G * dk, G * dv]
    offs = (8, 8 + widths[0] + -widths[0] % 8, 0)
    offs = (offs[0], offs[1], offs[1] + widths[1] + -widths[1] % 8)
    cols = max(dk, dv) + 8
    proj = rnd(T, offs[2] + widths[2] + 8).to(dt)
    slots = torch.randperm(8 * page)[:T]
    slots[5] = -1
    kc, vc = (torch.full((8, G, page, cols), 9.0, dtype=dt, device=dev) for _ in range(2))
    q = torch.full((T, H, cols), 7.0, dtype=dt, device=dev)
    ops.conv_qkv_prep(proj.to(dev), offs, H, G, dk, dv, None, None, None, None, ops.build_cos_sin(128, rot, base, device=dev),
                      i32(list(range(first, first + T)), dev), i32([0, T], dev), i32([0], dev), 1, T, slots.to(dev), kc, vc, q, 0.0)
    status_ok(dev)
    ok = slots >= 0
    for name, n, d, o, got in (("q", H, dk, offs[0], q), ("k", G, dk, offs[1], kc), ("v", G, dv, offs[2], vc)):
        for h in range(n):
            x = proj[:, o + h * d:o + (h + 1) * d].double()
            want = x if name == "v" else oracle.rotate_halves(x, base, rot, first)
            rows = got[:, h].cpu() if name == "q" else got[:, h].reshape(-1, cols).cpu()[slots[ok]]
            assert rel(rows[:, :d], want if name == "q" else want[ok]) < tol(dt)
            assert bool((rows[:, d:] == 0).all())
    untouched = torch.ones(8 * page, dtype=torch.bool)
    untouched[slots[ok]] = False
    assert bool((kc.transpose(1, 2).reshape(8 * page, -1).cpu()[untouched] == 9).all())


class Paged:
    """Random keys and values in shuffled pages, and the attention ops over them."""

    def __init__(self, target, H, G, D, page, ctxs, seed=0, scale_k=1.0):
        self.dev, self.dt = target
        self.H, self.G, self.D, self.page, self.ctxs, self.scale = H, G, D, page, ctxs, D ** -0.5
        self.rnd = gen(seed)
        mb = -(-max(ctxs) // page)
        n = mb * len(ctxs) + 3
        self.k, self.v = scale_k * self.rnd(n, G, page, D).to(self.dt), self.rnd(n, G, page, D).to(self.dt)
        self.tables = torch.randperm(n, generator=torch.Generator().manual_seed(seed))[:mb * len(ctxs)].view(len(ctxs), mb)

    def at(self, cache, b, i):
        return cache[self.tables[b, i // self.page], :, i % self.page]

    def run(self, q, q_lens, window, keep, decode):
        d = lambda t: t.to(self.dev)  # noqa: E731
        args = (d(q), d(self.k), d(self.v), d(self.tables.to(torch.int32)))
        ctx = i32(self.ctxs, self.dev)
        if decode:
            out = ops.attn_decode(*args, ctx, self.scale, window=window, max_ctx=max(self.ctxs), keep_first=keep)
        else:
            cu = i32([0] + torch.tensor(q_lens).cumsum(0).tolist(), self.dev)
            out = ops.attn_prefill(*args, cu, ctx, max(q_lens), self.scale, window=window, keep_first=keep)
        status_ok(self.dev)
        return out

    def want(self, q, q_lens, window, keep):
        out, t = torch.zeros(q.shape, dtype=torch.float64), 0
        for b, n in enumerate(q_lens):
            for h in range(self.H):
                k, v = (torch.stack([self.at(c, b, i)[h // (self.H // self.G)] for i in range(self.ctxs[b])]).double()
                        for c in (self.k, self.v))
                out[t:t + n, h] = oracle.attend(q[t:t + n, h].double(), k, v, self.scale, window or None, keep)
            t += n
        return out


SHAPES = [(3, 3, 24, 16), (6, 2, 64, 16), (8, 8, 128, 16), (40, 2, 64, 16), (4, 1, 200, 32), (4, 2, 128, 64)]


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,G,D,page", SHAPES)
@pytest.mark.parametrize("window,keep", [(20, 5), (64, 64), (70, 0), (30, 130), (1, 1), (0, 9), (129, 17)])
def test_windowed_attention_of_ragged_batches(target, H, G, D, page, window, keep):
    for q_lens, ctxs, decode in (([1, 1, 1, 1], [1, 17, 99, 330], True), ([9, 2, 1], [9, 67, 240], False), ([131], [300], False)):
        pg = Paged(target, H, G, D, page, ctxs, seed=H)
        q = pg.rnd(sum(q_lens), H, D).to(pg.dt)
        assert rel(pg.run(q, q_lens, window, keep, decode), pg.want(q, q_lens, window, keep)) < tol(pg.dt, 3e-6, 8e-3)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,G,D", [(2, 2, 24), (4, 2, 64), (4, 1, 128)])
@pytest.mark.parametrize("window,keep,ctx", [(40, 6, 180), (65, 64, 300), (100, 129, 400), (33, 1, 150)])
def test_one_key_stands_out(target, H, G, D, window, keep, ctx):
    """One key takes the whole softmax wherever it is visible: just inside and just outside the window of every query, the
    kept first tokens and the next ones, page and tile borders; prompts and decoding."""
    n = 70
    first, last = ctx - n, ctx - 1
    places = {0, keep - 1, keep, keep + 1, 15, 16, 63, 64, 127, 128, first - window, first - window + 1, first, last - window,
              last - window + 1, last - 1, last}
    for at in sorted(p for p in places if 0 <= p < ctx):
        pg = Paged(target, H, G, D, 16, [ctx], seed=at, scale_k=0.02)
        direction = pg.rnd(D)
        direction = direction / direction.norm()
        pg.at(pg.k, 0, at)[:] = (direction * 30).to(pg.dt)
        pg.at(pg.v, 0, at)[:] = 100.0
        q = (direction * 30).to(pg.dt).expand(n, H, D).contiguous()
        got = pg.run(q, [n], window, keep, False).float().mean((1, 2))
        one = float(pg.run(q[:1], [1], window, keep, True).float().mean())
        for i in range(n):
            assert (float(got[i]) > 90) == oracle.seen(first + i, at, window, keep), (at, first + i)
        assert (one > 90) == oracle.seen(last, at, window, keep), at


# ---------------------------------------------------------------------------------- matrix memory
def memory_inputs(rnd, T, H, dk, dv, dt, hard=False):
    offs = (8, 8 + H * dk + -(H * dk) % 8, 0)
    offs = (offs[0], offs[1], offs[1] + H * dk + -(H * dk) % 8)
    proj = rnd(T, offs[2] + H * dv + -(H * dv) % 8 + 8).to(dt)
    gates = torch.cat([3 * rnd(T, H), 3 * rnd(T, H), torch.full((T, 3), 99.0)], -1)
    bias = torch.cat([rnd(H), 2 + 2 * rnd(H)])
    if hard:       # gates at their caps: a forget gate that empties the memory, an input gate that drowns it, and the opposite
        gates[:, :2 * H] *= 10
        gates[::7, :H], gates[3::11, H:2 * H], gates[5::13, :H] = 60.0, -90.0, -90.0
    return offs, proj, gates, bias


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("plan", sorted(PLANS))
@pytest.mark.parametrize("H,dk,dv,cap,hard", [(2, 16, 24, 8.0, False), (3, 5, 7, 1.0, False), (1, 32, 32, 15.0, True), (2, 64, 96, 15.0, False),
                                              (2, 48, 40, 4.0, True), (1, 128, 136, 9.0, False), (1, 200, 64, 12.0, False),
                                              (1, 264, 33, 12.0, False)])
def test_matrix_memory(target, plan, H, dk, dv, cap, hard):
    """Slices of any size beside decoded tokens; dirty state slots; outputs and the state they leave behind."""
    dev, dt = target
    lens = [40, 3, 150]
    rnd = gen(H * dk + dv)
    offs, proj, gates, bias = memory_inputs(rnd, sum(lens), H, dk, dv, dt, hard)
    words = memory_words(dk, dv)
    state = torch.full((5, H, words), 30.0, device=dev)
    out = torch.zeros(sum(lens), H, dv)
    for rows, pos, cu, seqs, slices, _ in steps(lens, PLANS[plan]):
        got = ops.matrix_memory(proj[rows].to(dev), offs, H, dk, dv, gates[rows].to(dev), bias.to(dev), cap, state, i32(pos, dev),
                                i32(cu, dev), i32([4 - s for s in seqs], dev), slices, MEMORY_SLICE)
        out[rows] = got.float().cpu()
    status_ok(dev)
    slices = -(-dv // MEMORY_SLICE)
    for s, n in enumerate(lens):
        lo = sum(lens[:s])
        for h in range(H):
            q, k, v = (proj[lo:lo + n, o + h * d:o + (h + 1) * d].double() for o, d in zip(offs, (dk, dk, dv)))
            li = oracle.soft_cap(gates[lo:lo + n, h].double() + bias[h].double(), cap)
            lf = oracle.log_sigmoid(oracle.soft_cap(gates[lo:lo + n, H + h].double() + bias[H + h].double(), cap))
            want = oracle.matrix_memory(q / math.sqrt(dk), k, v, li, lf)
            got = out[lo:lo + n, h].double()
            err = (got - want).norm(dim=-1) / want.norm(dim=-1)
            assert float(err.median()) < tol(dt, 5e-6, 4e-3) and float(err.max()) < tol(dt, 3e-4, 6e-2), (s, h)
            # the state: sum over tokens of e^(F_n - F_t + i_t - m) k v^T, m = the largest exponent (or F_n)
            F = lf.cumsum(0)
            a = F[-1] - F + li
            m = max(float(a.max()), float(F[-1]))
            wgt = (a - m).exp()
            held = state[4 - s, h].double().cpu()
            close = dict(rtol=0, atol=1e-4 * float(wgt.sum().sqrt() + 1))
            assert torch.allclose(held[:dk * dv].view(dk, dv), (k * wgt[:, None]).T @ v, **close)
            for c in range(slices):
                assert torch.allclose(held[dk * dv + c * dk:dk * dv + (c + 1) * dk], (k * wgt[:, None]).sum(0), **close)
                assert abs(float(held[dk * dv + slices * dk + c]) - m) < 1e-4 * (1 + abs(m))


@pytest.mark.parametrize("target", TARGETS)
def test_a_far_token_is_remembered_or_forgotten(target):
    """One token writes a value that stands out; open forget gates keep it over hundreds of tokens, whichever way they are
    cut, and one closed gate in between drops it."""
    dev, dt = target
    H, dk, dv, T, cap = 1, 16, 32, 700, 15.0
    for at, closed in ((0, None), (1, None), (63, None), (64, 300), (5, 640)):
        rnd = gen(at)
        offs, proj, gates, bias = memory_inputs(rnd, T, H, dk, dv, dt)
        proj *= 0.05
        proj[:, offs[0]:offs[0] + dk] = 1.0                        # every query asks along the ones
        proj[at, offs[1]:offs[1] + dk], proj[at, offs[2]:offs[2] + dv] = 1.0, 50.0
        gates[:, :1], gates[:, 1:2], bias = -4.0, 40.0, torch.zeros(2)
        gates[at, 0] = 4.0
        if closed is not None:
            gates[closed, 1] = -40.0
        for cut in ([T], [at + 1, 1, 1, T - at - 3], [64, 65, 2, T - 131]):
            state = torch.full((2, H, memory_words(dk, dv)), -3.0, device=dev)
            lo, out = 0, []
            for n in cut:
                rows = slice(lo, lo + n)
                out.append(ops.matrix_memory(proj[rows].to(dev), offs, H, dk, dv, gates[rows].to(dev), bias.to(dev), cap, state,
                                             i32(list(range(lo, lo + n)), dev), i32([0, n], dev), i32([1], dev),
                                             int(n > 1 or lo == 0)).float().cpu())
                lo += n
            mean = torch.cat(out).mean((1, 2))
            assert float(mean[at]) > 20
            assert (float(mean[-1]) > 20) == (closed is None), (at, closed, cut)
            if closed is not None:
                assert float(mean[closed - 1]) > 20 and abs(float(mean[closed])) < 5
    status_ok(dev)


# ---------------------------------------------------------------------------------- heads, feed-forwards, token inputs
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,dv,cols", [(3, 5, 9), (4, 24, 24), (16, 64, 72), (2, 200, 200)])
def test_norm_per_head_gate_and_factor(target, H, dv, cols):
    dev, dt = target
    rnd, T, eps = gen(H * dv), 11, 1e-2
    x, gate, w = rnd(T, H, cols).to(dt), 2 * rnd(T, H * dv).to(dt), 1 + 0.3 * rnd(H * dv)
    x[3] *= 1e-3
    heads = [x[:, h, :dv].double() for h in range(H)]
    for norm in (True, False):
        out = torch.full((T, H * dv + 8 + -(H * dv) % 8), 5.0, dtype=dt, device=dev)
        ops.gated_rows(x.to(dev), dv, gate.to(dev), out, w.to(dev) if norm else None, eps, per_head=True, scale=0.37)
        want = torch.cat([oracle.over_rms(a, eps) for a in heads], -1) * w.double() if norm else torch.cat(heads, -1)
        assert rel(out[:, :H * dv], 0.37 * want * oracle.sigmoid(gate.double())) < tol(dt)
        assert bool((out[:, H * dv:] == 0).all())
    status_ok(dev)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("T,K,N", [(3, 30, 21), (5, 64, 40), (300, 128, 2048), (1300, 64, 512), (130, 256, 24)])
def test_activations_behind_a_product(target, T, K, N):
    """Few and many rows take different kernels; the table's row follows the token, its column block the layer."""
    dev, dt = target
    rnd = gen(T + N)
    x, w = rnd(T, K).to(dt), (rnd(N, K) / math.sqrt(K)).to(dt)
    table, ids = rnd(17, 3 * N).to(dt), torch.randint(0, 17, (T,), generator=torch.Generator().manual_seed(T))
    z = x.double() @ w.double().T
    assert rel(ops.act_linear(x.to(dev), w.to(dev), 3), oracle.relu_squared(z)) < tol(dt)
    got = ops.act_linear(x.to(dev), w.to(dev), 2, table.to(dev), i32(ids.tolist(), dev), N)
    assert rel(got, oracle.gelu_tanh(z) * table.double()[ids, N:2 * N]) < tol(dt)
    assert rel(ops.act_linear(x.to(dev), w.to(dev), 2), oracle.gelu_tanh(z)) < tol(dt)
    status_ok(dev)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("T,W,ff,E,top", [(7, 30, 11, 5, 3), (40, 64, 64, 6, 1), (150, 128, 72, 9, 4), (1, 48, 16, 4, 4)])
def test_experts_weighted_at_their_input(target, T, W, ff, E, top):
    """Sigmoid scores, not normalised, of either size: the gate's nonlinearity shows a weight at the wrong end."""
    from parallax_b200.models.layer_spec import ACT_SILU, GLUSpec, RoutedSpec
    from parallax_b200.models.moe import RoutedExperts

    dev, dt = target
    cfg = oracle.random_config([oracle.mlstm(mlp=oracle.moe(ff, E, top, shared=None))], width=W, side=0, loop=None)
    w, rnd = oracle.random_weights(cfg, seed=E), gen(T)
    spec = RoutedSpec(experts=E, identity=0, top=top, expert=GLUSpec(ff, ACT_SILU), sigmoid=True, correction=False,
                      normalised=False, shared_gate=False, weighted_input=True)
    get = lambda name, d=dt: w["l0.mlp." + name].to(device=dev, dtype=d)  # noqa: E731
    moe, h = RoutedExperts.build(spec, get, dev), (2 * rnd(T, W)).to(dt)
    picked = []
    moe.capture = lambda ids: picked.extend(ids.tolist())
    (rows, pos, wt), gate = moe.forward(h.to(dev))
    assert wt is None and gate is None
    got, record = rows[pos.view(T, top).long()][:, :, :W].double().sum(1).cpu(), []
    want = oracle.routed(cfg["layers"][0]["mlp"], w, "l0.mlp.", h.double(), record)
    same = [t for t in range(T) if set(picked[t]) == set(record[t])]       # (a close call may fall either way in bf16)
    assert len(same) >= (T if dt == torch.float32 else 0.9 * T)
    assert rel(got[same], want[same]) < tol(dt, 3e-6, 1e-2)
    status_ok(dev)


# ---------------------------------------------------------------------------------- errors are reported, not followed
@GPU
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_indices_outside_the_tables_are_reported(dt):
    from parallax_b200.ops import KernelError

    dev = "cuda:0"
    offs, proj, gates, bias = memory_inputs(gen(), 4, 1, 16, 24, dt)
    with pytest.raises(KernelError, match="index"):
        ops.matrix_memory(proj.cuda(), offs, 1, 16, 24, gates.cuda(), bias.cuda(), 5.0, torch.zeros(2, 1, memory_words(16, 24), device=dev),
                          i32(range(4), dev), i32([0, 4], dev), i32([77], dev), 1)
        status_ok(dev)
    for T in (4, 1300):
        x, w, table = torch.zeros(T, 64).to(dt).cuda(), torch.zeros(512, 64).to(dt).cuda(), torch.zeros(5, 512).to(dt).cuda()
        with pytest.raises(KernelError, match="row id"):
            ops.act_linear(x, w, 2, table, i32([99] * T, dev), 0)
            status_ok(dev)
    x = torch.zeros(2, 64, device=dev)
    with pytest.raises(KernelError, match="row id"):
        ops.residual_step(x, table=torch.ones(3, 64, device=dev, dtype=dt), ids=i32([1, -4], dev))
        status_ok(dev)
    assert float(x[0].sum()) == 64 and float(x[1].sum()) == 0
