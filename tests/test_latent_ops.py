"""Every mechanism of the Piburax layers alone: the op (CPU restatement or B200 kernel) against the equations in
``helpers/latent_oracle.py``, with inputs that make a single wrong key, sink, clip or table row stand out."""

import pytest
import torch

from helpers import latent_oracle as oracle
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


def tol(dt, f32=2e-6, bf16=6e-3):
    return f32 if dt == torch.float32 else bf16


def status_ok(dev):
    if dev != "cpu":
        from parallax_b200.ops import cuda as cu

        cu.check_status(torch.device(dev))


# ---------------------------------------------------------------------------------- embedding
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("bigram", [None, (13, 7, 3), (1, 5, 5), (65521, 2000003, 1000003)])
def test_embedding(target, bigram):
    dev, dt = target
    rnd = gen()
    cfg = oracle.random_config([], vocab=50000, width=24, emb_scale=2.5, bigram=bigram)
    w = {"embed": rnd(50000, 24).bfloat16()}
    if bigram:
        w["bigram"] = rnd(bigram[0] + 1, 24).bfloat16()
    toks = [49999, 49999, 0, 0, 12345, 49998]          # products beyond 32 bits with the large multipliers
    want = oracle.embedding(cfg, w, toks)
    ids = torch.tensor(toks, dtype=torch.int32, device=dev)
    prev = torch.tensor([-1] + toks[:-1], dtype=torch.int32, device=dev)
    args = (w["bigram"].to(dev, dt), prev, bigram[1], bigram[2], bigram[0]) if bigram else ()
    got = ops.embed_rows(w["embed"].to(dev, dt), ids, 2.5, *args)
    status_ok(dev)
    assert got.dtype == torch.float32 and rel(got, want) < 1e-6


# ---------------------------------------------------------------------------------- norms and the residual
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("width", [30, 48, 256, 4096, 20000])
def test_residual_norm(target, width):
    """Rows with a mean far above their deviation (a one-pass variance would lose them), and rows of tiny values (eps
    matters)."""
    dev, dt = target
    rnd = gen(width)
    x, w = rnd(5, width), 1 + 0.3 * rnd(width)
    y = rnd(5, width)
    y[1] = y[1] + (30 if dt == torch.bfloat16 else 300)
    y[2] *= 1e-3
    y = y.to(dt)
    for kind, norm in ((ops.NORM_LAYER, oracle.layer_norm), (ops.NORM_RMS, oracle.rms_norm)):
        xg = x.to(dev).clone()
        low = ops.residual_norm(xg, y.to(dev), w.to(dev), 1e-4, 0.7, kind)
        want = x.double() + 0.7 * norm(y.double(), w, 1e-4)
        assert rel(xg, want) < 3e-5 and low.dtype == dt
        assert rel(low, want) < tol(dt, 3e-5, 4e-3)


@pytest.mark.parametrize("target", TARGETS)
def test_norm_of_gathered_rows(target):
    dev, dt = target
    rnd = gen(3)
    x, w, rows = rnd(9, 96), rnd(96), torch.tensor([8, 0, 3, 3], dtype=torch.int32)
    got = ops.row_norm(x.to(dev), w.to(dev), 1e-6, rows=rows.to(dev), dtype=dt)
    status_ok(dev)
    assert got.dtype == dt and rel(got, oracle.layer_norm(x[rows.long()].double(), w, 1e-6)) < tol(dt)


# ---------------------------------------------------------------------------------- clipped GLU
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("rows,width,ff,limit", [(3, 64, 64, 0.5), (70, 128, 192, 1.3), (300, 256, 512, 7.0)])
def test_clipped_glu(target, rows, width, ff, limit):
    """Gates and ups on both sides of the clip; a gate far below zero is not clipped."""
    dev, dt = target
    rnd = gen(ff)
    x = rnd(rows, width).to(dt)
    gate, up = (rnd(ff, width) * 0.3).to(dt), (rnd(ff, width) * 0.3).to(dt)
    want = oracle.clip_and_gate(x.double() @ gate.double().T, x.double() @ up.double().T, limit)
    d = lambda t: t.to(dev)  # noqa: E731
    apart = ops.act_mul(ops.linear(d(x), d(torch.cat([gate, up]))), 1, limit)
    assert rel(apart, want) < tol(dt, 3e-6, 1e-2)
    if dt == torch.bfloat16 or dev == "cpu":
        fused = ops.linear(d(x), ops.interleave_gate_up(d(gate), d(up)), epi=ops.EPI_CLIP_GLU, limit=limit)
        assert rel(fused, want) < tol(dt, 3e-6, 5e-3)
    status_ok(dev)


# ---------------------------------------------------------------------------------- products
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("M,N,K", [(1, 8, 8), (3, 37, 19), (65, 130, 70), (200, 96, 256)])
def test_linear_of_any_shape(target, M, N, K):
    dev, dt = target
    rnd = gen(M)
    x, w = rnd(M, K).to(dt), rnd(N, K).to(dt)
    for epi in (ops.EPI_NONE, ops.EPI_F32):
        got = ops.linear(x.to(dev), w.to(dev), epi=epi)
        assert got.shape == (M, N) and rel(got, x.double() @ w.double().T) < tol(dt, 1e-6, 4e-3)
    status_ok(dev)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,K,N,pad,M", [(3, 7, 11, 2, 5), (4, 16, 40, 8, 33), (8, 128, 64, 64, 140), (2, 40, 264, 0, 300)])
def test_products_per_head_with_gate(target, heads, K, N, pad, M):
    """Head columns that do not fill a tile, neighbours of a head's columns that must not leak in, strided output."""
    dev, dt = target
    rnd = gen(K)
    hs = K + pad
    x, w, gate = rnd(M, heads * hs).to(dt), rnd(heads * N, K).to(dt), (2 * rnd(M, heads * N)).to(dt)
    plain = torch.stack([x[:, h * hs:h * hs + K].double() @ w[h * N:(h + 1) * N].double().T for h in range(heads)], 1)
    for g, want in ((None, plain), (gate, plain * torch.sigmoid(gate.double().view(M, heads, N)))):
        buf = torch.full((M, heads, N + 8), 5.0, dtype=dt, device=dev)
        ops.head_linear(x.to(dev), hs, w.to(dev), heads, buf[:, :, :N], None if g is None else g.to(dev))
        assert rel(buf[:, :, :N], want) < tol(dt, 1e-6, 4e-3)
        assert bool((buf[:, :, N:] == 5).all())
    status_ok(dev)


# ---------------------------------------------------------------------------------- cache rows and rotation
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,dim,R,rot,latent", [(3, 5, 6, 6, 19), (4, 16, 8, 8, 40), (2, 8, 24, 16, 64)])
def test_cache_rows_and_query_rotation(target, heads, dim, R, rot, latent):
    """Positions far apart, a row without a slot, rotated parts with a tail that passes unchanged."""
    dev, dt = target
    rnd = gen(latent)
    T, first, base = 6, 900, 321.0
    width = heads * (dim + R)
    proj = rnd(T, width + latent + R + 3).to(dt)
    norm_w = 1 + 0.3 * rnd(latent)
    table = ops.build_cos_sin(1000, rot, base)
    pos = torch.arange(first, first + T, dtype=torch.int32)
    slots = torch.tensor([30, 2, -1, 17, 0, 47])
    cache = torch.full((3, 1, 16, latent + R), 9.0, dtype=dt, device=dev)
    q_cat = torch.zeros((T, heads, latent + R), dtype=dt, device=dev)
    d = lambda t: t.to(dev)  # noqa: E731
    ops.latent_prep(d(proj), width, heads, dim + R, dim, d(norm_w), d(table), d(pos), d(slots), cache, q_cat, 1e-5, latent, R, rot)
    status_ok(dev)
    p = proj.double()
    c = oracle.rms_norm(p[:, width:width + latent], norm_w, 1e-5)
    k = oracle.rotate(p[:, width + latent:width + latent + R], base, rot, first)
    flat = cache.view(48, latent + R)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert rel(flat[s], torch.cat([c[t], k[t]])) < tol(dt)
    untouched = [i for i in range(48) if i not in slots.tolist()]
    assert bool((flat[untouched] == 9).all())
    for h in range(heads):
        q = oracle.rotate(p[:, h * (dim + R) + dim:(h + 1) * (dim + R)], base, rot, first)
        assert rel(q_cat[:, h, latent:], q) < tol(dt)


# ---------------------------------------------------------------------------------- attention over pages
class Paged:
    """Sequences of cached rows on shuffled pages, with helpers to run and to restate attention."""

    def __init__(self, target, H, latent, R, page, ctxs, seed=0, scale_rows=0.5):
        self.dev, self.dt = target
        self.H, self.L, self.D, self.page, self.ctxs = H, latent, latent + R, page, ctxs
        self.rnd = gen(seed)
        pages = [-(-c // page) for c in ctxs]
        n = sum(pages) + 3
        perm = torch.randperm(n, generator=torch.Generator().manual_seed(seed))
        self.tables, o = torch.zeros(len(ctxs), max(pages), dtype=torch.int32), 0
        for i, k in enumerate(pages):
            self.tables[i, :k] = perm[o:o + k].int()
            o += k
        self.cache = (self.rnd(n, 1, page, self.D) * scale_rows).to(self.dt)
        self.scale = 1.3 * self.D ** -0.5

    def row(self, b, pos):
        return self.cache.view(-1, self.D)[int(self.tables[b, pos // self.page]) * self.page + pos % self.page]

    def rows(self, b):
        return torch.stack([self.row(b, i) for i in range(self.ctxs[b])]).double()

    def run(self, q, q_lens, window, sinks, decode):
        d = lambda t: None if t is None else t.to(self.dev)  # noqa: E731
        cu = None if decode else torch.tensor([0] + torch.tensor(q_lens).cumsum(0).tolist(), dtype=torch.int32)
        out = ops.latent_attn(d(q), d(self.cache), d(self.tables), d(cu), d(torch.tensor(self.ctxs, dtype=torch.int32)),
                              self.scale, self.L, window, d(sinks), max(q_lens), max(self.ctxs))
        status_ok(self.dev)
        return out

    def want(self, q, q_lens, window, sinks):
        out, t = [], 0
        for b, n in enumerate(q_lens):
            kv = self.rows(b)
            ctx = self.ctxs[b]
            mask = oracle.window_mask(ctx, window or ctx)[ctx - n:]
            for i in range(n):
                heads = []
                for h in range(self.H):
                    s = (kv @ q[t, h].double() * self.scale).masked_fill(~mask[i], float("-inf"))[None]
                    sink = float("-inf") if sinks is None else sinks[h]
                    p = torch.softmax(s, -1) if sinks is None else oracle.softmax_with_sink(s, sink)
                    heads.append((p @ kv[:, :self.L])[0])
                out.append(torch.stack(heads))
                t += 1
        return torch.stack(out)


SIZES = [(3, 40, 8, 16), (5, 19, 6, 16), (8, 128, 64, 32), (32, 512, 64, 16), (130, 264, 56, 16), (12, 320, 64, 64), (64, 64, 16, 16)]


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,latent,R,page", SIZES)
@pytest.mark.parametrize("window", [0, 1, 33])
def test_attention_of_ragged_batches(target, H, latent, R, page, window):
    for q_lens, ctxs, decode in (([1, 1, 1, 1], [1, 16, 34, 150], True), ([9, 2, 1], [9, 67, 40], False)):
        pg = Paged(target, H, latent, R, page, ctxs, seed=H)
        q = pg.rnd(sum(q_lens), H, pg.D).to(pg.dt)
        for sinks in (None, 2 * pg.rnd(H)):
            got = pg.run(q, q_lens, window, sinks, decode)
            assert rel(got, pg.want(q, q_lens, window, sinks)) < tol(pg.dt, 3e-6, 8e-3)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,latent,R", [(3, 40, 8), (4, 128, 32), (32, 512, 64)])
@pytest.mark.parametrize("window", [20, 33, 64, 129])
def test_one_key_stands_out(target, H, latent, R, window):
    """One cached row matches the query so well that it takes the whole softmax when it is visible: planted just inside
    and just outside the window, at page and tile borders, at the first token - in decoding and in a prompt."""
    ctx = 180
    last = ctx - 1
    for at in sorted({0, 1, last, last - 1, last - window + 1, last - window, last - window - 1, 15, 16, 63, 64, 127, 128}):
        if not 0 <= at <= last:
            continue
        pg = Paged(target, H, latent, R, 16, [ctx], seed=at, scale_rows=0.02)
        q = pg.rnd(1, H, pg.D)
        q = q / q.norm(dim=-1, keepdim=True)
        row = pg.row(0, at)
        row.copy_((q[0].mean(0) / q[0].mean(0).norm() * 40).to(pg.dt))        # in place: a view of the cache
        q = (q * 40).to(pg.dt)
        sinks = torch.zeros(H)
        for q_lens, qq in (([1], q), ([7], torch.cat([q] * 7))):      # the prompt's last seven tokens ask the same
            got = pg.run(qq, q_lens, window, sinks, len(q_lens) == 1 and q_lens[0] == 1)
            want = pg.want(qq, q_lens, window, sinks)
            big = float(row[:latent].double().norm())
            for i in range(q_lens[0]):
                pos = last - q_lens[0] + 1 + i
                seen = at <= pos and pos - at < window
                assert (float(got[i].double().cpu().norm(dim=-1).max()) > 0.3 * big) == seen, (at, pos)
                assert float((got[i].double().cpu() - want[i]).norm()) < 0.02 * big


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,latent,R", [(3, 40, 8), (4, 128, 32)])
def test_sinks(target, H, latent, R):
    """A large sink takes nearly all the mass, a very negative one none; they are not scaled and count once whatever the
    number of keys, tiles or pages; the first token of a sequence has only itself and the sink."""
    for ctx in (1, 5, 150):
        pg = Paged(target, H, latent, R, 16, [ctx], seed=ctx)
        q = pg.rnd(1, H, pg.D).to(pg.dt)
        for value in (-1e4, -3.0, 0.0, 4.0, 12.0):
            sinks = torch.full((H,), value)
            sinks[0] = 0.5
            got, want = pg.run(q, [1], 0, sinks, True), pg.want(q, [1], 0, sinks)
            for h in range(H):
                assert rel(got[:, h], want[:, h]) < tol(pg.dt, 5e-6, 1e-2), (ctx, value, h)


@pytest.mark.parametrize("target", TARGETS)
def test_scores_that_grow_along_the_keys(target):
    """Ever larger scores move the running maximum in every tile (a stale rescale would show), and ever smaller ones never."""
    for sign in (1, -1):
        pg = Paged(target, 4, 128, 32, 16, [300], seed=7, scale_rows=0.3)
        q = torch.zeros(6, 4, pg.D)
        q[:, :, 0] = 30.0
        for i in range(300):
            pg.row(0, i)[0] = sign * i / 8.0
        q = q.to(pg.dt)
        for q_lens, qq, decode in (([6], q, False), ([1], q[:1], True)):
            got, want = pg.run(qq, q_lens, 0, torch.zeros(4), decode), pg.want(qq, q_lens, 0, torch.zeros(4))
            assert rel(got, want) < tol(pg.dt, 1e-5, 1e-2)


@pytest.mark.parametrize("target", TARGETS)
def test_rows_do_not_depend_on_their_neighbours(target):
    """A query's result is the same bits alone and in a batch, and on other pages."""
    H, latent, R = 4, 128, 32
    pg = Paged(target, H, latent, R, 16, [70, 200, 33], seed=5)
    q = pg.rnd(3, H, pg.D).to(pg.dt)
    whole = pg.run(q, [1, 1, 1], 50, None, True)
    for b in range(3):
        alone = Paged(target, H, latent, R, 16, [pg.ctxs[b]], seed=99)
        for i in range(pg.ctxs[b]):
            alone.row(0, i).copy_(pg.row(b, i))
        assert torch.equal(alone.run(q[b:b + 1], [1], 50, None, True)[0], whole[b])


@GPU
def test_bad_table_entry_is_reported_not_followed():
    from parallax_b200.ops import KernelError

    for target in (("cuda:0", torch.float32), ("cuda:0", torch.bfloat16)):
        pg = Paged(target, 4, 128, 32, 16, [40])
        pg.tables[0, 1] = 10 ** 6
        with pytest.raises(KernelError, match="block"):
            pg.run(pg.rnd(1, 4, pg.D).to(pg.dt), [1], 0, None, True)
