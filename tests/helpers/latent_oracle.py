"""Plain, slow restatement of the Piburax layers for the tests: one function per mechanism, whole sequences at once,
expanded per-head keys and values (no absorbed products, no cache, no pages), float64. Nothing here is shared with
the product path; weights are the checkpoint-named tensors."""

import math

import torch


def random_config(layers, vocab=83, width=48, eps=1e-6, mult=0.35, emb_scale=1.7, bigram=(61, 19, 5)):
    """``layers``: dicts with heads, dim, rot_dim, vdim, kv_rank, scale, window, base, ff (None: no feed-forward),
    limit."""
    out = []
    for d in layers:
        out.append({"type": "latent_attention",
                    "mixer": {"heads": d["heads"], "dim": d["dim"], "rot_dim": d["rot_dim"], "vdim": d["vdim"],
                              "kv_rank": d["kv_rank"], "scale": d["scale"], "mask": {"size": d["window"]},
                              "rot": {"base": d["base"], "dims": d["rot_dim"]}},
                    "mlp": None if d.get("ff") is None else {"kind": "dense", "ff": d["ff"], "limit": d["limit"]}})
    cfg = {"architecture": "Piburax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
           "embedding": {"scale": emb_scale, "bigram": None}, "layers": out}
    if bigram:
        cfg["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return cfg


def random_weights(cfg, seed=0):
    """bf16 tensors whose sublayers all matter: unit-scale projections, sinks and gates of either sign, norm weights
    around 1, clipped activations on both sides."""
    g = torch.Generator().manual_seed(seed)

    def lin(n, k, s=1.0):
        return (torch.randn(n, k, generator=g) * s / math.sqrt(k)).bfloat16()

    def near_one(n):
        return (1 + 0.2 * torch.randn(n, generator=g)).bfloat16()

    W, w = cfg["width"], {}
    w["embed"] = torch.randn(cfg["vocab"], W, generator=g).bfloat16()
    if cfg["embedding"]["bigram"]:
        w["bigram"] = torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, W, generator=g).bfloat16()
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        H = m["heads"]
        w[p + "norm1"] = near_one(W)
        w[p + "mix.q"] = lin(H * (m["dim"] + m["rot_dim"]), W, 1.5)
        w[p + "mix.dkv"] = lin(m["kv_rank"] + m["rot_dim"], W)
        w[p + "mix.dkv.norm"] = near_one(m["kv_rank"])
        w[p + "mix.uk"] = lin(H * m["dim"], m["kv_rank"])
        w[p + "mix.uv"] = lin(H * m["vdim"], m["kv_rank"])
        w[p + "mix.sink"] = (1.5 * torch.randn(H, generator=g)).bfloat16()
        w[p + "mix.g"] = lin(H * m["vdim"], W, 1.5)
        w[p + "mix.o"] = lin(W, H * m["vdim"])
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            w[p + "norm2"] = near_one(W)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff)
    w["final.norm"] = near_one(W)
    w["head"] = lin(cfg["vocab"], W)
    return w


def embedding(cfg, w, tokens):
    e = cfg["embedding"]
    rows = []
    for i, t in enumerate(tokens):
        x = w["embed"][t].double() * e["scale"]
        if e["bigram"]:
            b = e["bigram"]
            k = b["buckets"] if i == 0 else (tokens[i - 1] * b["mul_prev"] + t * b["mul_cur"]) % b["buckets"]
            x = x + w["bigram"][k].double()
        rows.append(x)
    return torch.stack(rows)


def layer_norm(x, weight, eps):
    mean = x.sum(-1, keepdim=True) / x.shape[-1]
    dev = x - mean
    var = (dev * dev).sum(-1, keepdim=True) / x.shape[-1]
    return dev / (var + eps).sqrt() * weight.double()


def rms_norm(x, weight, eps):
    return x / ((x * x).sum(-1, keepdim=True) / x.shape[-1] + eps).sqrt() * weight.double()


def rotate(x, base, dims, first=0):
    """x [T, R]: row p is rotated to position ``first + p``, pair (2i, 2i + 1) by angle position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = (first + torch.arange(x.shape[0], dtype=torch.float64)) * base ** (-2.0 * i / dims)
        u, v = x[:, 2 * i], x[:, 2 * i + 1]
        out[:, 2 * i] = u * a.cos() - v * a.sin()
        out[:, 2 * i + 1] = v * a.cos() + u * a.sin()
    return out


def softmax_with_sink(scores, sink):
    """scores [T, S] with -inf where hidden; the sink takes its share of the mass."""
    top = torch.maximum(scores.max(-1, keepdim=True).values, torch.full((1, 1), float(sink), dtype=torch.float64))
    e = (scores - top).exp()
    return e / (e.sum(-1, keepdim=True) + (float(sink) - top).exp())


def window_mask(n, size):
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (i >= j) & (i - j < size)


def latent_attention(m, w, p, x, eps):
    H, d, r, v, L = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    f = lambda name: w[p + "mix." + name].double()  # noqa: E731
    q = x @ f("q").T
    down = x @ f("dkv").T
    c = rms_norm(down[:, :L], w[p + "mix.dkv.norm"], eps)
    k_rot = rotate(down[:, L:], m["rot"]["base"], m["rot"]["dims"])
    keys, values = c @ f("uk").T, c @ f("uv").T
    keep = window_mask(x.shape[0], m["mask"]["size"])
    heads = []
    for h in range(H):
        qh = q[:, h * (d + r):(h + 1) * (d + r)]
        q_rot = rotate(qh[:, d:], m["rot"]["base"], m["rot"]["dims"])
        s = (qh[:, :d] @ keys[:, h * d:(h + 1) * d].T + q_rot @ k_rot.T) * m["scale"]
        s = s.masked_fill(~keep, float("-inf"))
        heads.append(softmax_with_sink(s, w[p + "mix.sink"][h]) @ values[:, h * v:(h + 1) * v])
    gated = torch.cat(heads, -1) / (1 + (-(x @ f("g").T)).exp())
    return gated @ f("o").T


def clip_and_gate(gate, up, limit):
    g, u = gate.clamp(max=limit), up.clamp(-limit, limit)
    return g / (1 + (-1.702 * g).exp()) * (u + 1)


def clipped_glu(mlp, w, p, x):
    f = lambda name: w[p + "mlp." + name].double()  # noqa: E731
    return clip_and_gate(x @ f("gate").T, x @ f("up").T, mlp["limit"]) @ f("down").T


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] (float64)."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embedding(cfg, w, tokens)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + mult * layer_norm(latent_attention(layer["mixer"], w, p, x, eps), w[p + "norm1"], eps)
        if layer["mlp"]:
            x = x + mult * layer_norm(clipped_glu(layer["mlp"], w, p, x), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["head"].double().T


def greedy(cfg, w, prompt, n):
    seq, margins = list(prompt), []
    for _ in range(n):
        top = forward(cfg, w, seq)[-1].topk(2)
        seq.append(int(top.indices[0]))
        margins.append(float(top.values[0] - top.values[1]))
    return seq[len(prompt):], margins
