"""Every mechanism of Kikurax alone, ``ops`` on CPU (fp32) and on a B200 (fp32, bf16) against the plain functions of
``helpers/kikurax_oracle.py`` in float64, with inputs made so that one key, one decay or one position decides."""

import math

import pytest
import torch

from helpers import kikurax_oracle as oracle
from parallax_b200 import ops

GPU = pytest.mark.gpu
TARGETS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda:0", torch.float32), id="gpu-fp32", marks=GPU),
           pytest.param(("cuda:0", torch.bfloat16), id="gpu-bf16", marks=GPU)]


class Maker:
    """Random tensors in the target's dtype; ``f64`` gives exactly what the kernels read."""

    def __init__(self, target, seed=0):
        self.dev, self.dt = target
        self.g = torch.Generator().manual_seed(seed)

    def rnd(self, *shape, s=1.0):
        return (torch.randn(*shape, generator=self.g) * s).to(self.dt).to(self.dev)

    def f32(self, *shape, s=1.0, at=0.0):
        return (torch.randn(*shape, generator=self.g) * s + at).to(self.dev)

    def i32(self, x):
        return torch.tensor(x, dtype=torch.int32, device=self.dev)


def f64(t):
    return t.double().cpu()


def near(got, want, target, what="", f32=2e-5, bf16=8e-3):
    """Largest difference, in units of the largest wanted value."""
    d = float((f64(got) - want).abs().max() / want.abs().max().clamp_min(1e-30))
    assert d < (f32 if target[1] == torch.float32 else bf16), (what, d)


class Pages:
    """A paged cache whose pages lie in no order, with rubbish in pages that nobody holds."""

    def __init__(self, mk, heads, cols, lens, page=16):
        per = [-(-n // page) for n in lens]
        total = sum(per) + 3
        order = torch.randperm(total, generator=mk.g).tolist()
        self.k, self.v = (mk.rnd(total, heads, page, cols, s=5.0) for _ in range(2))
        self.tables = torch.full((len(lens), max(per)), -1, dtype=torch.int32)
        for b, n in enumerate(per):
            self.tables[b, :n] = torch.tensor([order.pop() for _ in range(n)])
        self.page, self.tables = page, self.tables.to(mk.dev)

    def slots(self, b, lo, hi):
        pos = torch.arange(lo, hi)
        return self.tables[b].cpu()[pos // self.page].long() * self.page + pos % self.page

    def fill(self, b, k, v):
        """k, v [n, heads, cols]"""
        s = self.slots(b, 0, k.shape[0])
        self.k[s // self.page, :, s % self.page] = k
        self.v[s // self.page, :, s % self.page] = v


# ---------------------------------------------------------------------------------- attention weights
SIZES = [(4, 2, 64), (8, 8, 128), (12, 1, 128), (20, 1, 64), (3, 3, 40)]


def score_kw(mode, mk, H):
    if mode == "sink":
        return dict(sinks=torch.zeros(H, device=mk.dev))
    if mode == "capped":
        return dict(sinks=torch.zeros(H, device=mk.dev), softcap=2.5)
    return dict(sigmoid_bias=mk.f32(H, s=1.5, at=-2.0))


def plain_attention(mode, kw, q, k, v, scale):
    """q [T, H, D], k, v [T, G, D] -> [T, H, D]: every query over the keys up to its own place."""
    H, G, out = q.shape[1], k.shape[1], []
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * scale
        if mode == "capped":
            s = oracle.softcap(s, kw["softcap"])
        w = oracle.sigmoid_weights(s, f64(kw["sigmoid_bias"])[h]) if mode == "sigmoid" else oracle.sink_weights(s)
        out.append(w @ v[:, h // (H // G)])
    return torch.stack(out, 1)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("mode", ["sink", "capped", "sigmoid"])
@pytest.mark.parametrize("H,G,D", SIZES)
def test_attention_weights_of_prompts_and_decoding(mode, H, G, D, target):
    """Unequal sequences, prefixes, page borders; one far key whose score stands out, and queries that see little."""
    mk, lens, new, scale = Maker(target, H * 10 + G), [150, 17, 300, 64, 1], [150, 1, 130, 33, 1], 0.3
    pages, kw, qs, want = Pages(mk, G, D, lens), score_kw(mode, mk, H), [], []
    for b, (n, m) in enumerate(zip(lens, new)):
        q, k, v = mk.rnd(n, H, D, s=D ** -0.25), mk.rnd(n, G, D, s=D ** -0.25), mk.rnd(n, G, D)
        k[n // 3] = (q[-1, ::H // G][:G].float() * 3).to(k.dtype)        # the last query's far key
        v[n // 3] = 4.0
        pages.fill(b, k, v)
        qs.append(q[n - m:])
        want.append(plain_attention(mode, kw, f64(q), f64(k), f64(v), scale)[n - m:])
    cu = mk.i32([0] + torch.tensor(new).cumsum(0).tolist())
    got = ops.attn_prefill(torch.cat(qs), pages.k, pages.v, pages.tables, cu, mk.i32(lens), max(new), scale, **kw)
    near(got, torch.cat(want), target, "prompt", f32=5e-6, bf16=1e-2)
    last = torch.stack([q[-1] for q in qs])
    got = ops.attn_decode(last, pages.k, pages.v, pages.tables, mk.i32(lens), scale, max_ctx=max(lens), **kw)
    near(got, torch.stack([w[-1] for w in want]), target, "decoded", f32=5e-6, bf16=1e-2)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("mode", ["capped", "sigmoid"])
@pytest.mark.parametrize("D", [64, 128, 24])
def test_attention_weights_over_a_long_context(mode, D, target):
    """Decoding in splits that are added up: keys in every one, one of them far back and heavy."""
    mk, n, H, G = Maker(target, D), 2500, 4, 2
    pages, kw = Pages(mk, G, D, [n]), score_kw(mode, mk, H)
    q, k, v = mk.rnd(1, H, D), mk.rnd(n, G, D, s=0.3), mk.rnd(n, G, D)
    k[5] = (q[0, ::2].float() * 2).to(k.dtype)
    pages.fill(0, k, v)
    got = ops.attn_decode(q, pages.k, pages.v, pages.tables, mk.i32([n]), D ** -0.5, max_ctx=n, **kw)
    full = torch.cat([torch.zeros(n - 1, H, D, dtype=torch.float64), f64(q)])
    near(got, plain_attention(mode, kw, full, f64(k), f64(v), D ** -0.5)[-1:], target, f32=5e-6, bf16=1e-2)


@pytest.mark.parametrize("target", TARGETS)
def test_a_soft_cap_and_sigmoids_at_their_ends(target):
    """Scores far beyond the cap, weights next to 0 and 1: nothing overflows."""
    mk, n, H = Maker(target, 5), 70, 2
    for D in (64, 128):
        pages = Pages(mk, H, D, [n])
        q, k, v = mk.rnd(n, H, D, s=12.0), mk.rnd(n, H, D, s=12.0), mk.rnd(n, H, D)
        pages.fill(0, k, v)
        for mode, kw in (("capped", dict(sinks=torch.zeros(H, device=mk.dev), softcap=6.0)),
                         ("sigmoid", dict(sigmoid_bias=torch.tensor([-90.0, 30.0], device=mk.dev)))):
            got = ops.attn_prefill(q, pages.k, pages.v, pages.tables, mk.i32([0, n]), mk.i32([n]), n, 1.0, **kw)
            near(got, plain_attention(mode, kw, f64(q), f64(k), f64(v), 1.0), target, mode, f32=2e-5, bf16=1e-2)


# ---------------------------------------------------------------------------------- queries, keys and values
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,G,dk,dv,cols,rot", [(4, 2, 64, 48, 64, 64), (6, 3, 96, 128, 128, 32), (5, 5, 7, 5, 16, 4), (8, 1, 128, 64, 128, 0),
                                               (2, 1, 200, 136, 200, 16), (3, 1, 24, 16, 64, 6)])
def test_heads_norms_rotation_temperatures_and_mixed_values(H, G, dk, dv, cols, rot, target):
    mk, T, eps, page = Maker(target, dk + dv), 37, 1e-4, 16
    widths, offs, at = (H * dk, G * dk, G * dv), [], 8
    for w in widths:
        offs.append(at)
        at += w + -w % 8
    proj = mk.rnd(T, at + 8)
    first = mk.rnd(T, G * dv + 8)[:, :G * dv]
    pos = torch.randint(0, 90, (T,), generator=mk.g).int().to(mk.dev)
    table = ops.build_cos_sin(100, rot, 500.0, device=mk.dev) if rot else None
    head_scale, pos_scale = mk.f32(H, at=1.0), (1 + 0.3 * torch.arange(100).float()).to(mk.dev)
    slots = torch.randperm(5 * page, generator=mk.g)[:T].to(mk.dev)
    slots[3] = -1                                                     # a row that belongs to no page
    k, v = (torch.full((5, G, page, cols), 9.0, dtype=mk.dt, device=mk.dev) for _ in range(2))
    q = torch.empty(T, H, cols, dtype=mk.dt, device=mk.dev)
    ops.head_qkv_prep(proj, tuple(offs), H, G, dk, dv, eps, table, pos, slots, k, v, q, head_scale, pos_scale, first, 0.3)

    def heads(o, n, d):
        x = f64(proj[:, o:o + n * d]).view(T, n, d)
        return x

    def rotated(x):
        if not rot:
            return x
        freq = torch.tensor([500.0 ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
        a = f64(pos)[:, None, None] * freq
        u, w = x[..., :rot // 2], x[..., rot // 2:rot]
        return torch.cat([u * torch.cos(a) - w * torch.sin(a), w * torch.cos(a) + u * torch.sin(a), x[..., rot:]], -1)

    pad = torch.nn.functional.pad
    wq = oracle.over_rms(rotated(heads(offs[0], H, dk)), eps) * f64(head_scale)[:, None] * f64(pos_scale)[f64(pos).long()][:, None, None]
    wk = oracle.over_rms(rotated(heads(offs[1], G, dk)), eps)
    wv = 0.7 * heads(offs[2], G, dv) + 0.3 * f64(first).reshape(T, G, dv)
    near(q, pad(wq, (0, cols - dk)), target, "q", bf16=5e-3)
    keep = slots >= 0
    s = slots[keep]
    near(k[s // page, :, s % page], pad(wk, (0, cols - dk))[keep.cpu()], target, "k", bf16=5e-3)
    near(v[s // page, :, s % page], pad(wv, (0, cols - dv))[keep.cpu()], target, "v", bf16=5e-3)
    assert int((k == 9.0).all(-1).sum()) >= (5 * page - T) * G


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("C,taps,bias", [(64, 4, True), (1032, 2, False), (13, 5, True), (24, 1, True), (2048, 3, True), (40, 8, False)])
def test_short_convolutions(C, taps, bias, target):
    """Portions down to one token, decoded rows beside them, state slots that held something else; a far channel's spike is
    seen for exactly ``taps`` tokens."""
    mk, n = Maker(target, C + taps), 90
    w, b = mk.rnd(taps, C), mk.rnd(C) if bias else None
    state = torch.full((6, max(taps - 1, 1), C), 33.0, dtype=mk.dt, device=mk.dev) if taps > 1 else None
    seqs, want = [mk.rnd(n, C + 8) for _ in range(3)], []
    for x in seqs:
        x[20] += 50.0
        want.append(oracle.short_conv(f64(x[:, :C]), f64(w).T, None if b is None else f64(b)))
    at, slot, got = [0, 0, 0], [4, 0, 2], [[], [], []]
    for step in ([70, 1, 2], [2, 1, 1], [1, 50, 3], [1, 38, 84], [16, 0, 0]):
        prompts = [i for i in range(3) if step[i] > 1]
        single = [i for i in range(3) if step[i] == 1]
        order = prompts + single
        rows = torch.cat([seqs[i][at[i]:at[i] + step[i]] for i in order])
        cu = torch.tensor([0] + [step[i] for i in order]).cumsum(0).tolist()
        pos = torch.cat([torch.arange(at[i], at[i] + step[i]) for i in order]).int().to(mk.dev)
        out = ops.short_conv(rows[:, :C], w, b, state, pos, mk.i32(cu), mk.i32([slot[i] for i in order]), len(prompts),
                             sum(step[i] for i in prompts))
        for j, i in enumerate(order):
            got[i].append(out[cu[j]:cu[j + 1]])
            at[i] += step[i]
    assert at == [n, n, n]
    for i in range(3):
        near(torch.cat(got[i]), want[i], target, i, bf16=5e-3)
    if state is not None:
        assert bool((state[[1, 3, 5]] == 33.0).all())
        near(state[4], f64(seqs[0][n - taps + 1:, :C]), target)


# ---------------------------------------------------------------------------------- recurrences
def run_steps(op, seqs, steps, slots, dev):
    """Feed three sequences of rows through ``op(rows, positions, cu, slots, prompts, tokens)``, returns each one's output."""
    at, got = [0] * len(seqs), [[] for _ in seqs]
    for step in steps:
        prompts = [i for i in range(len(seqs)) if step[i] > 1]
        order = prompts + [i for i in range(len(seqs)) if step[i] == 1]
        if not order:
            continue
        rows = [torch.cat([s[at[i]:at[i] + step[i]] for i, s in ((i, seqs[i][part]) for i in order)]) for part in range(len(seqs[0]))]
        cu = torch.tensor([0] + [step[i] for i in order]).cumsum(0).tolist()
        pos = torch.cat([torch.arange(at[i], at[i] + step[i]) for i in order]).int().to(dev)
        out = op(*rows, pos, torch.tensor(cu, dtype=torch.int32, device=dev),
                 torch.tensor([slots[i] for i in order], dtype=torch.int32, device=dev), len(prompts), sum(step[i] for i in prompts))
        for j, i in enumerate(order):
            got[i].append(out[cu[j]:cu[j + 1]])
            at[i] += step[i]
    return [torch.cat(g) for g in got]


STEPS = ([130, 2, 1], [1, 64, 63], [2, 1, 65], [37, 65, 1], [1, 1, 40], [3, 41, 4])


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,Hk,dk,dv,decays", [
    (2, 2, 64, 32, "mixed"), (4, 2, 128, 128, "mixed"), (3, 1, 32, 72, "mixed"), (2, 1, 16, 24, "mixed"), (6, 3, 9, 7, "mixed"),
    (1, 1, 96, 40, "mixed"), (1, 1, 264, 8, "mixed"), *((*size, d) for size in ((4, 2, 128, 128), (2, 1, 16, 24))
                                                       for d in ("none", "slow", "fast"))])
def test_delta_rule(H, Hk, dk, dv, decays, target):
    """Portions beside single tokens, states that are carried; decays per channel from none to a factor of 1e-30 a token."""
    mk = Maker(target, H * dk + dv)
    at = {"none": -30.0, "slow": -6.0, "mixed": -1.0, "fast": 4.0}[decays]
    qo, ko, vo = 0, Hk * dk + -(Hk * dk) % 8, 2 * (Hk * dk + -(Hk * dk) % 8)
    C = vo + H * dv + -(H * dv) % 8
    dt_bias, A_log = mk.f32(H * dk, s=2.0 if decays == "mixed" else 0.3, at=at), mk.f32(H, s=1.0 if decays == "mixed" else 0.2)
    if decays == "fast":
        A_log += 2.5
    state = torch.full((5, H, dk, dv), 7.0, device=mk.dev)
    n = 174
    seqs = [(mk.rnd(n, C), mk.f32(n, H * dk + 8), mk.f32(n, H + 3, s=2.0)) for _ in range(3)]
    seqs[0][0][100:103, ko:ko + Hk * dk] = 0              # a key of zeros is no unit vector
    for i in range(60, 64):                               # one key again and again: the rule replaces its value
        seqs[1][0][i, ko:ko + Hk * dk] = seqs[1][0][60, ko:ko + Hk * dk]

    def op(x, decay, beta, pos, cu, slots, prompts, tokens):
        return ops.delta_rule(x, (qo, ko, vo), H, Hk, dk, dv, decay, dt_bias, A_log, beta, state, pos, cu, slots, prompts, tokens)

    got = run_steps(op, seqs, STEPS, [3, 0, 4], mk.dev)
    for i, (x, decay, beta) in enumerate(seqs):
        q, k, v = (oracle.heads_of(f64(x[:, o:o + c * d]), c, d) for o, c, d in ((qo, Hk, dk), (ko, Hk, dk), (vo, H, dv)))
        dt = oracle.heads_of(oracle.softplus(f64(decay[:, :H * dk]) + f64(dt_bias)), H, dk)
        b, rep = oracle.sigmoid(f64(beta)), H // Hk
        want = torch.stack([oracle.delta_rule(oracle.unit(q[h // rep]) / math.sqrt(dk), oracle.unit(k[h // rep]), v[h], b[:, h],
                                              -torch.exp(f64(A_log)[h]) * dt[h]) for h in range(H)], 1)
        near(got[i], want, target, i, f32=2e-5, bf16=6e-3)
    assert bool((state[[1, 2]] == 7.0).all()) and not bool((state[[0, 3, 4]] == 7.0).all())


@pytest.mark.gpu
def test_delta_rule_chunks_agree_with_single_tokens():
    """The same bf16 rows as one prompt (chunks, in several runs over the workspace) and in 32-bit token by token: states to
    1e-4, outputs to their rounding."""
    target = ("cuda:0", torch.bfloat16)
    mk, H, d, n = Maker(target, 3), 32, 128, 4700
    x, decay, beta = mk.rnd(n, 3 * H * d), mk.f32(n, H * d), mk.f32(n, H, s=2.0)
    dt_bias, A_log = mk.f32(H * d, s=2.0, at=-3.0), mk.f32(H, s=1.0)
    cu, pos = mk.i32([0, 4000, 4001, n]), torch.cat([torch.arange(m) for m in (4000, 1, n - 4001)]).int().to("cuda:0")
    slots, res = mk.i32([2, 0, 1]), []
    for dt in (torch.bfloat16, torch.float32):
        state = torch.full((3, H, d, d), 7.0, device="cuda:0")
        out = ops.delta_rule(x.to(dt), (0, H * d, 2 * H * d), H, H, d, d, decay, dt_bias, A_log, beta, state, pos, cu, slots, 3, n)
        res.append((f64(out), f64(state)))
    near(res[0][1], res[1][1], ("cuda:0", torch.float32), "state", f32=1e-4)
    near(res[0][0], res[1][0], target, "out", bf16=5e-3)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("at", [-20.0, -3.0, 3.0])
@pytest.mark.parametrize("H,G,N,dv", [(4, 2, 64, 32), (6, 1, 128, 64), (2, 2, 32, 72), (3, 3, 5, 7), (4, 1, 256, 40), (2, 1, 300, 8)])
def test_state_space(H, G, N, dv, at, target):
    mk = Maker(target, H * N + dv)
    xo, bo, co = 0, H * dv + -(H * dv) % 8, H * dv + -(H * dv) % 8 + G * N + -(G * N) % 8
    C = co + G * N + -(G * N) % 8
    dt_bias, A_log, D = mk.f32(H, s=1.0, at=at), mk.f32(H), mk.f32(H, at=1.0)
    state, n = torch.full((5, H, N, dv), 7.0, device=mk.dev), 174
    seqs = [(mk.rnd(n, C), mk.f32(n, H + 5)) for _ in range(3)]
    seqs[2][0][7, bo:co] *= 20                            # a token that stays in the state

    def op(x, dt, pos, cu, slots, prompts, tokens):
        return ops.state_space(x, (xo, bo, co), H, G, N, dv, dt, dt_bias, A_log, D, state, pos, cu, slots, prompts)

    got = run_steps(op, seqs, STEPS, [3, 0, 4], mk.dev)
    for i, (x, dt) in enumerate(seqs):
        v, B, c = (oracle.heads_of(f64(x[:, o:o + m * d]), m, d) for o, m, d in ((xo, H, dv), (bo, G, N), (co, G, N)))
        d, rep = oracle.softplus(f64(dt[:, :H]) + f64(dt_bias)), H // G
        want = torch.stack([oracle.state_space(v[h], B[h // rep], c[h // rep], d[:, h], torch.exp(f64(A_log))[h], f64(D)[h])
                            for h in range(H)], 1)
        near(got[i], want, target, i, f32=2e-5, bf16=6e-3)
    assert bool((state[[1, 2]] == 7.0).all())


# ---------------------------------------------------------------------------------- norms, residual, experts
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,vdim,groups", [(4, 64, 1), (8, 64, 8), (6, 40, 3), (5, 7, 5), (3, 8, 2), (32, 128, 16), (64, 8, 4)])
def test_gate_before_a_grouped_norm(heads, vdim, groups, target):
    mk, T, eps, n = Maker(target, heads), 19, 1e-3, heads * vdim
    x, gate, w = mk.rnd(T, heads, vdim), mk.rnd(T, n + 8, s=2.0), mk.f32(n, at=1.0)
    x[:, 0] *= 100                                        # one part far larger than the others
    out = torch.full((T, n + -n % 8 + 8), 5.0, dtype=mk.dt, device=mk.dev)
    ops.gated_norm_rows(x, gate[:, :n], w, groups, eps, out)
    y = f64(x).reshape(T, n) * oracle.silu(f64(gate[:, :n]))
    near(out[:, :n], oracle.grouped_norm(y, f64(w), eps, groups), target, bf16=5e-3)
    assert bool((out[:, n:] == 0).all())


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("W,groups", [(64, 1), (256, 4), (30, 5), (72, 9), (2048, 8), (4096, 16), (24, 2), (10240, 2)])
def test_residual_updates_and_grouped_norms(W, groups, target):
    """One update, two normed updates, expert rows, each followed by the grouped norm; norms of gathered rows."""
    mk, T, eps, k = Maker(target, W), 11, 1e-4, 3
    x0, w, w1, w2 = mk.f32(T, W), mk.f32(W, at=1.0), mk.f32(W, at=1.0), mk.f32(W, at=1.0)
    x0[:, :W // groups] *= 50
    y1, y2, rows = mk.rnd(T, W), mk.rnd(T, W, s=9.0), mk.rnd(T * k + 4, W + -W % 8 + 8)
    pos = torch.randperm(T * k + 4, generator=mk.g)[:T * k].view(T, k).int().to(mk.dev)
    shares = torch.rand(T, k, generator=mk.g).to(mk.dev)

    def norm(x, n):
        return oracle.grouped_norm(x, f64(n), eps, groups)

    def check(add, want, what, **kw):
        for last in (w, None):
            x = x0.clone()
            low = ops.residual_add(x, add, last, eps, groups=groups, **kw)
            near(x, want, ("", torch.float32), what, f32=3e-6)
            if last is None:
                assert low is None
            else:
                assert low.dtype == mk.dt
                near(low, norm(want, w), target, what, f32=5e-6, bf16=5e-3)

    check(y1, f64(x0) + f64(y1), "one")
    both = (oracle.over_rms(f64(y1), eps) * f64(w1) + oracle.over_rms(f64(y2), eps) * f64(w2)) * 0.5
    check(None, f64(x0) + both, "two", branches=(0.5, (y1, w1), (y2, w2)))
    picked = (f64(rows)[f64(pos).long()][:, :, :W] * f64(shares)[:, :, None]).sum(1)
    check(None, f64(x0) + picked, "experts", routed=(rows, pos, shares), h=y1)
    ids = mk.i32([3, 0, 10, 3])
    near(ops.row_norm(x0, w, eps, ops.NORM_RMS, rows=ids, dtype=mk.dt, groups=groups), norm(f64(x0)[f64(ids).long()], w), target, bf16=5e-3)
    assert ops.row_norm(x0, w, eps, ops.NORM_RMS, rows=ids[:0], dtype=mk.dt, groups=groups).shape == (0, W)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("W,ff,experts,top,limit", [(64, 64, 4, 1, 0.4), (128, 96, 12, 3, 2.0), (30, 11, 5, 5, 1.0), (256, 200, 40, 8, 7.0)])
def test_routed_experts_with_clips_and_biases(W, ff, experts, top, limit, target):
    """The bias decides which experts are chosen; activations beyond the clip on both sides."""
    from parallax_b200.models.layer_spec import parse_layers
    from parallax_b200.models.moe import RoutedExperts

    mk, T = Maker(target, W + ff), 33
    cfg = oracle.moe(ff, experts, top, limit)
    spec = parse_layers("Kikurax", [oracle.mamba2(mlp=cfg)])[0].mlp
    w = {"router": mk.rnd(experts, W, s=W ** -0.5), "router.b": mk.rnd(experts, s=8.0)}
    for e in range(experts):
        w.update({f"e{e}.gate": mk.rnd(ff, W, s=3 * W ** -0.5), f"e{e}.up": mk.rnd(ff, W, s=3 * W ** -0.5),
                  f"e{e}.down": mk.rnd(W, ff, s=ff ** -0.5)})
    moe = RoutedExperts.build(spec, lambda n, dt=mk.dt: w[n].to(dt), mk.dev)
    h, record, ids = mk.rnd(T, W), [], []
    moe.capture = ids.append
    x = torch.zeros(T, W, device=mk.dev)
    routed, gate = moe.forward(h)
    ops.residual_add(x, None, None, 0.0, routed, h)
    want = oracle.routed(cfg, {k: t.cpu() for k, t in w.items()}, "", f64(h), record)
    assert gate is None and [sorted(r) for r in ids[0].tolist()] == [sorted(r) for r in record]
    near(x, want, target, f32=1e-5, bf16=1e-2)
