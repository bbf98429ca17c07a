"""Plain, slow restatement of the Zudepel layers for the tests: one function per mechanism, whole sequences at once
(no cache, no pages, no carried state), float64. Nothing here is shared with the product path; weights are the
checkpoint-named tensors."""

import math

import torch


# ---------------------------------------------------------------------------------- configurations and weights
def lightning(heads=3, dim=16, vdim=8, decay=None, mlp=None):
    decay = decay or [math.exp(-2.0 ** -(h % 4)) if h % 3 else 0.998 for h in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def attention(heads=4, kv_heads=2, dim=24, vdim=16, conv=4, rot=16, base=1000.0, scale=0.2, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale,
         "rot": {"dims": rot, "base": base}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=6, top=2, identity=2, groups=(4, 2), shared=32):
    router = {"experts": experts, "top": top, "identity": identity}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def random_config(layers, vocab=83, width=48, eps=1e-6):
    return {"architecture": "Zudepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def random_weights(cfg, seed=0):
    """bf16 tensors whose sublayers all matter: unit-scale projections, biases, sinks, corrections and gates of
    either sign, norm weights around 1, convolutions that look back as much as they look at the token itself."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0):
        return (torch.randn(*shape, generator=g) * s).bfloat16()

    def lin(n, k, s=1.0):
        return rnd(n, k, s=s / math.sqrt(k))

    def near_one(n):
        return (1 + 0.2 * torch.randn(n, generator=g)).bfloat16()

    W, w = cfg["width"], {}
    w["embed"] = rnd(cfg["vocab"], W)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        w[p + "norm1"] = near_one(W)
        out = m["heads"] * m["vdim"]
        if layer["type"] == "lightning":
            w[p + "mix.q"], w[p + "mix.k"] = lin(m["heads"] * m["dim"], W, 1.5), lin(m["heads"] * m["dim"], W, 1.5)
            w[p + "mix.v"], w[p + "mix.norm"] = lin(out, W, 1.5), near_one(out)
        else:
            rows = {"q": m["heads"] * m["dim"]}
            if m.get("kv_from") is None:
                rows.update(k=m["kv_heads"] * m["dim"], v=m["kv_heads"] * m["vdim"])
            for name, n in rows.items():
                w[p + f"mix.{name}"], w[p + f"mix.{name}.b"] = lin(n, W), rnd(n, s=0.4)
                w[p + f"mix.{name}.conv"] = rnd(n, m["conv"], s=0.6)
                if name != "v":
                    w[p + f"mix.{name}.norm"] = near_one(n)
            w[p + "mix.sink"] = rnd(m["heads"], s=1.5)
        w[p + "mix.g"], w[p + "mix.o"] = lin(out, W, 1.5), lin(W, out)
        mlp = layer["mlp"]
        if mlp is None:
            continue

        def ffn(q, ff):
            w[q + "gate"], w[q + "up"], w[q + "down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff)

        p += "mlp."
        if mlp["kind"] == "dense":
            ffn(p, mlp["ff"])
            continue
        r = mlp["router"]
        E = r["experts"] + (r.get("identity") or 0)
        for e in range(r["experts"]):
            ffn(p + f"e{e}.", mlp["expert"]["ff"])
        w[p + "router"], w[p + "correction"] = lin(E, W), rnd(E, s=0.1)
        if mlp.get("shared"):
            ffn(p + "shared.", mlp["shared"]["ff"])
            w[p + "shared.sg"] = lin(1, W, 1.5)
    w["final.norm"] = near_one(W)
    w["head"] = lin(cfg["vocab"], W)
    return w


# ---------------------------------------------------------------------------------- small pieces
def sigmoid(x):
    return 1 / (1 + (-x).exp())


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1 + (math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)).tanh())


def rms_norm(x, weight, eps):
    return x / ((x * x).sum(-1, keepdim=True) / x.shape[-1] + eps).sqrt() * weight.double()


def glu(x, gate, up, down, act):
    return (act(x @ gate.double().T) * (x @ up.double().T)) @ down.double().T


# ---------------------------------------------------------------------------------- lightning attention
def decayed_sum(q, k, v, decay):
    """One head: o_t = sum over j <= t of decay^(t - j) (q_t . k_j) v_j, written as the sum (no recurrence)."""
    n = q.shape[0]
    out = torch.zeros(n, v.shape[1], dtype=torch.float64)
    for t in range(n):
        back = torch.arange(t, -1, -1, dtype=torch.float64)
        out[t] = ((k[:t + 1] @ q[t]) * decay ** back) @ v[:t + 1]
    return out


def lightning_mixer(m, w, p, h, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    f = lambda name: w[p + "mix." + name].double()  # noqa: E731
    q, k, v = (silu(h @ f(n).T) for n in "qkv")
    heads = [decayed_sum(q[:, i * d:(i + 1) * d], k[:, i * d:(i + 1) * d], v[:, i * dv:(i + 1) * dv], m["decay"][i])
             for i in range(H)]
    return (rms_norm(torch.cat(heads, -1), f("norm"), eps) * sigmoid(h @ f("g").T)) @ f("o").T


# ---------------------------------------------------------------------------------- attention
def causal_conv(u, taps):
    """u [T, C], taps [C, K]: the last tap meets the token itself."""
    T, K = u.shape[0], taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(K):
            s = t - K + 1 + j
            if s >= 0:
                y[t] += taps[:, j].double() * u[s]
    return y


def rotate_half(x, base, dims, first=0):
    """x [T, D]: row p is rotated to position ``first + p``, pair (i, i + dims / 2) by position * base^(-2i / dims)."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        a = (first + torch.arange(x.shape[0], dtype=torch.float64)) * base ** (-2.0 * i / dims)
        u, v = x[:, i], x[:, i + half]
        out[:, i] = u * a.cos() - v * a.sin()
        out[:, i + half] = v * a.cos() + u * a.sin()
    return out


def softmax_with_sink(scores, sink):
    """scores [T, S] with -inf where hidden; the sink takes its share of the mass."""
    top = torch.maximum(scores.max(-1, keepdim=True).values, torch.full((1, 1), float(sink), dtype=torch.float64))
    e = (scores - top).exp()
    return e / (e.sum(-1, keepdim=True) + (float(sink) - top).exp())


def projection(w, p, name, h):
    """Projection, bias, convolution."""
    u = h @ w[p + f"mix.{name}"].double().T + w[p + f"mix.{name}.b"].double()
    return causal_conv(u, w[p + f"mix.{name}.conv"])


def split_heads(x, n, dim):
    return [x[:, i * dim:(i + 1) * dim] for i in range(n)]


def rotated_heads(m, w, p, name, n, h, eps):
    x = rms_norm(projection(w, p, name, h), w[p + f"mix.{name}.norm"], eps)
    return [rotate_half(a, m["rot"]["base"], m["rot"]["dims"]) for a in split_heads(x, n, m["dim"])]


def attend(q, keys, values, scale, sink):
    T = q.shape[0]
    hidden = torch.ones(T, T, dtype=torch.bool).triu(1)
    return softmax_with_sink((q @ keys.T * scale).masked_fill(hidden, float("-inf")), sink) @ values


def attention_mixer(m, w, p, h, eps, shared_kv):
    """``shared_kv``: layer index -> (keys, values) of the layers before; a layer of its own adds its pair."""
    H, G = m["heads"], m["kv_heads"]
    q = rotated_heads(m, w, p, "q", H, h, eps)
    if m.get("kv_from") is None:
        kv = rotated_heads(m, w, p, "k", G, h, eps), split_heads(projection(w, p, "v", h), G, m["vdim"])
        shared_kv[int(p[1:-1])] = kv
    else:
        kv = shared_kv[m["kv_from"]]
    heads = [attend(q[i], kv[0][i // (H // G)], kv[1][i // (H // G)], m["scale"], w[p + "mix.sink"][i]) for i in range(H)]
    return (torch.cat(heads, -1) * sigmoid(h @ w[p + "mix.g"].double().T)) @ w[p + "mix.o"].double().T


# ---------------------------------------------------------------------------------- feed-forwards
def choose(scores, correction, top, groups):
    """Ids of the experts of one token: scores [E] (softmax), correction [E]."""
    choice = [float(s) + float(c) for s, c in zip(scores, correction)]
    E = len(choice)
    if groups:
        size = E // groups["count"]
        best = sorted(range(groups["count"]), key=lambda g: -max(choice[g * size:(g + 1) * size]))[:groups["keep"]]
        choice = [c if e // size in best else -math.inf for e, c in enumerate(choice)]
    return sorted(range(E), key=lambda e: -choice[e])[:top]


def router_scores(logits):
    e = (logits - logits.max()).exp()
    return e / e.sum()


def routed(mlp, w, p, h, record=None):
    r, n = mlp["router"], mlp["router"]["experts"]
    out = torch.zeros_like(h)
    z = h @ w[p + "router"].double().T
    for t in range(h.shape[0]):
        s = router_scores(z[t])
        ids = choose(s, w[p + "correction"].double(), r["top"], r.get("groups"))
        if record is not None:
            record.append(ids)
        total = sum(float(s[e]) for e in ids) + 1e-20
        for e in ids:
            x = h[t:t + 1]
            y = x if e >= n else glu(x, w[p + f"e{e}.gate"], w[p + f"e{e}.up"], w[p + f"e{e}.down"], silu)
            out[t] += float(s[e]) / total * y[0]
    if mlp.get("shared"):
        y = glu(h, w[p + "shared.gate"], w[p + "shared.up"], w[p + "shared.down"], silu)
        out = out + y * sigmoid(h @ w[p + "shared.sg"].double().T)
    return out


def feed_forward(mlp, w, p, h):
    p += "mlp."
    if mlp["kind"] == "dense":
        return glu(h, w[p + "gate"], w[p + "up"], w[p + "down"], gelu_tanh)
    return routed(mlp, w, p, h)


# ---------------------------------------------------------------------------------- the model
def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] (float64)."""
    eps, shared_kv = cfg["norm"]["eps"], {}
    x = w["embed"][torch.tensor(tokens)].double()
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "lightning":
            y = lightning_mixer(layer["mixer"], w, p, h, eps)
        else:
            y = attention_mixer(layer["mixer"], w, p, h, eps, shared_kv)
        if layer["mlp"] is not None:
            y = y + feed_forward(layer["mlp"], w, p, h)
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].double().T


def greedy(cfg, w, prompt, n):
    seq, margins = list(prompt), []
    for _ in range(n):
        top = forward(cfg, w, seq)[-1].topk(2)
        seq.append(int(top.indices[0]))
        margins.append(float(top.values[0] - top.values[1]))
    return seq[len(prompt):], margins
