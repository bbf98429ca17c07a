"""Plain, slow restatement of the Zasalix layers for the tests: one function per mechanism, whole sequences at once
(no cache, no pages, no carried state), float64. Nothing here is shared with the product path; weights are the
checkpoint-named tensors."""

import math

import torch


# ---------------------------------------------------------------------------------- configurations
def latent(heads=3, dim=16, rot_dim=8, vdim=12, kv_rank=24, q_rank=20, base=1000.0, rot=None, scale=0.2, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "scale": scale, "rot": {"base": base, "dims": rot or rot_dim}}}


def memory(heads=2, dim=16, vdim=24, cap=9.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def mlstm(heads=2, dim=16, vdim=24, cap=9.0, mlp=None):
    return {"type": "mlstm", "mixer": memory(heads, dim, vdim, cap), "mlp": mlp}


def windowed(heads=4, kv_heads=2, dim=24, vdim=16, rot=16, base=1000.0, scale=0.2, size=20, keep=5):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
            "rot": {"base": base, "dims": rot}, "mask": {"size": size, "keep_first": keep}}


def parallel(left=None, right=None, scales=(0.7, 0.4), mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left or windowed(), "right": right or memory(),
                                                      "left_scale": scales[0], "right_scale": scales[1]}}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=6, top=2, shared=32):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def random_config(layers, vocab=83, width=48, eps=1e-5, side=10, loop=(0, 1, 2)):
    cfg = {"architecture": "Zasalix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    if side:
        cfg["token_side"] = {"dim": side}
    return cfg


# ---------------------------------------------------------------------------------- weights
def random_weights(cfg, seed=0):
    """bf16 tensors whose sublayers all matter: norms that bend without saturating, sinks and gates of either sign,
    forget gates from short to long memory, steps of the loop and token inputs as large as a sublayer's output."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0):
        return (torch.randn(*shape, generator=g) * s).bfloat16()

    def lin(n, k, s=1.0):
        return rnd(n, k, s=s / math.sqrt(k))

    def near_one(n):
        return (1 + 0.2 * torch.randn(n, generator=g)).bfloat16()

    W, w = cfg["width"], {}

    def tanh_norm(name, alpha):
        w[name], w[name + ".b"] = near_one(W), rnd(W, s=0.1)
        w[name + ".alpha"] = torch.tensor(alpha * (1 + 0.3 * float(torch.rand(1, generator=g)))).bfloat16()

    def memory_weights(p, m):
        for name in "qk":
            w[p + name] = lin(m["heads"] * m["dim"], W, 1.5)
        out = m["heads"] * m["vdim"]
        w[p + "v"], w[p + "g"], w[p + "o"], w[p + "norm"] = lin(out, W), lin(out, W, 1.5), lin(W, out), near_one(out)
        w[p + "i"], w[p + "i.b"] = lin(m["heads"], W, 2.0), rnd(m["heads"])
        w[p + "f"], w[p + "f.b"] = lin(m["heads"], W, 1.5), (3 + 2 * torch.randn(m["heads"], generator=g)).bfloat16()

    w["embed"] = rnd(cfg["vocab"], W)
    if cfg.get("loop"):
        w["loop.step"] = rnd(cfg["loop"]["times"], W, s=0.5)
    side = (cfg.get("token_side") or {}).get("dim")
    if side:
        w["side.embed"] = rnd(cfg["vocab"], len(cfg["layers"]) * side)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        tanh_norm(p + "norm1", 0.6)
        tanh_norm(p + "norm1b", 0.9)
        if layer["mlp"] is not None:
            tanh_norm(p + "norm2", 0.5)
            tanh_norm(p + "norm2b", 0.9)
        q = p + "mix."
        if layer["type"] == "latent_attention":
            H = m["heads"]
            w[q + "dq"], w[q + "dq.norm"] = lin(m["q_rank"], W), near_one(m["q_rank"])
            w[q + "uq"] = lin(H * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.5)
            w[q + "dkv"], w[q + "dkv.norm"] = lin(m["kv_rank"] + m["rot_dim"], W, 1.5), near_one(m["kv_rank"])
            w[q + "uk"], w[q + "uv"] = lin(H * m["dim"], m["kv_rank"], 1.5), lin(H * m["vdim"], m["kv_rank"], 1.5)
            w[q + "sink"], w[q + "o"] = rnd(H, s=1.5), lin(W, H * m["vdim"])
        elif layer["type"] == "mlstm":
            memory_weights(q, m)
        else:
            a = m["left"]
            w[q + "left.q"], w[q + "left.k"] = lin(a["heads"] * a["dim"], W, 1.5), lin(a["kv_heads"] * a["dim"], W, 1.5)
            w[q + "left.v"], w[q + "left.g"] = lin(a["kv_heads"] * a["vdim"], W, 1.5), lin(a["heads"] * a["vdim"], W, 1.5)
            w[q + "left.o"] = lin(W, a["heads"] * a["vdim"], 1.5)
            memory_weights(q + "right.", m["right"])
        if side:
            w[p + "side.gate"], w[p + "side.proj"], w[p + "side.norm"] = lin(side, W), lin(W, side), near_one(W)
        mlp, q = layer["mlp"], p + "mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            w[q + "up"], w[q + "down"] = lin(mlp["ff"], W, 1.5), lin(W, mlp["ff"])
            continue

        def expert(n, ff):
            w[q + n + "gate"], w[q + n + "up"], w[q + n + "down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff, 1.5)

        for e in range(mlp["router"]["experts"]):
            expert(f"e{e}.", mlp["expert"]["ff"])
        w[q + "router"] = lin(mlp["router"]["experts"], W, 2.0)
        if mlp.get("shared"):
            expert("shared.", mlp["shared"]["ff"])
    tanh_norm("final.norm", 0.7)
    w["head"] = lin(cfg["vocab"], W)
    return w


# ---------------------------------------------------------------------------------- small pieces
def sigmoid(x):
    return 1 / (1 + (-x).exp())


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1 + (math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)).tanh())


def relu_squared(x):
    return x.clamp_min(0) ** 2


def over_rms(x, eps):
    return x / ((x * x).sum(-1, keepdim=True) / x.shape[-1] + eps).sqrt()


def tanh_norm(x, w, name):
    return (w[name + ".alpha"].double() * x).tanh() * w[name].double() + w[name + ".b"].double()


def heads_of(x, n, dim):
    return [x[:, i * dim:(i + 1) * dim] for i in range(n)]


def angles(T, base, dims, i, first=0):
    return (first + torch.arange(T, dtype=torch.float64)) * base ** (-2.0 * i / dims)


def turned(u, v, a):
    return u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()


def rotate_neighbours(x, base, dims):
    """x [T, D], row p at position p: pairs (2i, 2i + 1)."""
    out = x.clone()
    for i in range(dims // 2):
        out[:, 2 * i], out[:, 2 * i + 1] = turned(x[:, 2 * i], x[:, 2 * i + 1], angles(x.shape[0], base, dims, i))
    return out


def rotate_halves(x, base, dims, first=0):
    """x [T, D], row p at position ``first + p``: pairs (i, i + dims / 2)."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        out[:, i], out[:, i + half] = turned(x[:, i], x[:, i + half], angles(x.shape[0], base, dims, i, first))
    return out


def softmax_rows(scores, sink=None):
    """scores [T, S], -inf where hidden; a sink takes its share of the mass."""
    top = scores.max(-1, keepdim=True).values
    if sink is not None:
        top = top.clamp_min(float(sink))
    e = (scores - top).exp()
    total = e.sum(-1, keepdim=True)
    return e / (total if sink is None else total + (float(sink) - top).exp())


def seen(i, j, size=None, keep=0):
    """Whether the query at ``i`` sees the key at ``j``."""
    return j <= i and (size is None or i - j < size or j < keep)


def attend(q, keys, values, scale, size=None, keep=0, sink=None):
    T, S = q.shape[0], keys.shape[0]
    hidden = torch.tensor([[not seen(S - T + i, j, size, keep) for j in range(S)] for i in range(T)])
    return softmax_rows((q @ keys.T * scale).masked_fill(hidden, float("-inf")), sink) @ values


# ---------------------------------------------------------------------------------- latent attention
def latent_mixer(m, w, p, h, eps):
    f = lambda name: w[p + name].double()  # noqa: E731
    H, R, rot = m["heads"], m["rot_dim"], m["rot"]
    q = (over_rms(h @ f("dq").T, eps) * f("dq.norm")) @ f("uq").T
    down = h @ f("dkv").T
    c = over_rms(down[:, :m["kv_rank"]], eps) * f("dkv.norm")
    shared = rotate_neighbours(down[:, m["kv_rank"]:], rot["base"], rot["dims"])
    up_k, up_v, out = heads_of(c @ f("uk").T, H, m["dim"]), heads_of(c @ f("uv").T, H, m["vdim"]), []
    for i, qi in enumerate(heads_of(q, H, m["dim"] + R)):
        turned_q = rotate_neighbours(qi[:, m["dim"]:], rot["base"], rot["dims"])
        out.append(attend(torch.cat([qi[:, :m["dim"]], turned_q], -1), torch.cat([up_k[i], shared], -1), up_v[i], m["scale"],
                          sink=f("sink")[i]))
    return torch.cat(out, -1) @ f("o").T


# ---------------------------------------------------------------------------------- windowed attention
def windowed_mixer(m, w, p, h):
    f = lambda name: w[p + name].double()  # noqa: E731
    H, G, rot, mask = m["heads"], m["kv_heads"], m["rot"], m.get("mask") or {}
    q, k = ([rotate_halves(x, rot["base"], rot["dims"]) for x in heads_of(h @ f(n).T, c, m["dim"])] for n, c in (("q", H), ("k", G)))
    v = heads_of(h @ f("v").T, G, m["vdim"])
    out = [attend(q[i], k[i // (H // G)], v[i // (H // G)], m["scale"], mask.get("size"), mask.get("keep_first") or 0)
           for i in range(H)]
    return (torch.cat(out, -1) * sigmoid(h @ f("g").T)) @ f("o").T


# ---------------------------------------------------------------------------------- matrix memory
def soft_cap(z, cap):
    return cap * (z / cap).tanh()


def log_sigmoid(z):
    return -torch.nn.functional.softplus(-z)


def matrix_memory(q, k, v, log_in, log_forget):
    """One head, token by token: q, k [T, d], v [T, dv], gates [T] (logarithms). Returns [T, dv]."""
    S, n, m, out = torch.zeros(k.shape[1], v.shape[1], dtype=torch.float64), torch.zeros(k.shape[1], dtype=torch.float64), 0.0, []
    for t in range(q.shape[0]):
        top = max(float(log_forget[t]) + m, float(log_in[t]))
        keep, take = math.exp(float(log_forget[t]) + m - top), math.exp(float(log_in[t]) - top)
        S = keep * S + take * k[t][:, None] * v[t][None, :]
        n = keep * n + take * k[t]
        m = top
        out.append(S.T @ q[t] / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6))
    return torch.stack(out)


def memory_mixer(m, w, p, h, eps):
    f = lambda name: w[p + name].double()  # noqa: E731
    H, cap = m["heads"], m["gate_cap"]
    log_in, log_forget = soft_cap(h @ f("i").T + f("i.b"), cap), log_sigmoid(soft_cap(h @ f("f").T + f("f.b"), cap))
    q, k, v = heads_of(h @ f("q").T / math.sqrt(m["dim"]), H, m["dim"]), heads_of(h @ f("k").T, H, m["dim"]), \
        heads_of(h @ f("v").T, H, m["vdim"])
    out = [over_rms(matrix_memory(q[i], k[i], v[i], log_in[:, i], log_forget[:, i]), eps) for i in range(H)]
    return (torch.cat(out, -1) * f("norm") * sigmoid(h @ f("g").T)) @ f("o").T


def mixer(layer, w, p, h, eps):
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        return latent_mixer(m, w, p, h, eps)
    if layer["type"] == "mlstm":
        return memory_mixer(m, w, p, h, eps)
    return m["left_scale"] * windowed_mixer(m["left"], w, p + "left.", h) + \
        m["right_scale"] * memory_mixer(m["right"], w, p + "right.", h, eps)


# ---------------------------------------------------------------------------------- feed-forwards
def expert(x, w, p):
    return (silu(x @ w[p + "gate"].double().T) * (x @ w[p + "up"].double().T)) @ w[p + "down"].double().T


def chosen(scores, top):
    return sorted(range(len(scores)), key=lambda e: -float(scores[e]))[:top]


def routed(mlp, w, p, h, record=None):
    scores = sigmoid(h @ w[p + "router"].double().T)
    out = expert(h, w, p + "shared.") if mlp.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = chosen(scores[t], mlp["router"]["top"])
        if record is not None:
            record.append(ids)
        for e in ids:
            out[t] += expert(scores[t][e] * h[t:t + 1], w, p + f"e{e}.")[0]
    return out


def feed_forward(mlp, w, p, h):
    if mlp["kind"] == "dense":
        return relu_squared(h @ w[p + "up"].double().T) @ w[p + "down"].double().T
    return routed(mlp, w, p, h)


# ---------------------------------------------------------------------------------- the model
def token_input(cfg, w, i, x, tokens):
    """What layer ``i`` adds for its token's row of the side table."""
    d, p = cfg["token_side"]["dim"], f"l{i}.side."
    e = w["side.embed"][torch.tensor(tokens), i * d:(i + 1) * d].double()
    y = (gelu_tanh(x @ w[p + "gate"].double().T) * e) @ w[p + "proj"].double().T
    return over_rms(y, cfg["norm"]["eps"]) * w[p + "norm"].double()


def run_layer(cfg, w, i, x, tokens):
    layer, p = cfg["layers"][i], f"l{i}."
    x = x + tanh_norm(mixer(layer, w, p + "mix.", tanh_norm(x, w, p + "norm1"), cfg["norm"]["eps"]), w, p + "norm1b")
    if layer["mlp"] is not None:
        x = x + tanh_norm(feed_forward(layer["mlp"], w, p + "mlp.", tanh_norm(x, w, p + "norm2")), w, p + "norm2b")
    return x + token_input(cfg, w, i, x, tokens) if cfg.get("token_side") else x


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] (float64); ``layers_out`` collects the residual after every run of a layer."""
    first = x = w["embed"][torch.tensor(tokens)].double()
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 0}
    n = len(cfg["layers"])

    def run(span, x):
        for i in span:
            x = run_layer(cfg, w, i, x, tokens)
            if layers_out is not None:
                layers_out.append(x)
        return x

    x = run(range(loop["start"]), x)
    for t in range(loop["times"]):
        if t:
            x = x + first
        x = run(range(loop["start"], loop["stop"]), x + w["loop.step"][t].double())
    x = run(range(loop["stop"], n), x)
    return tanh_norm(x, w, "final.norm") @ w["head"].double().T


def greedy(cfg, w, prompt, n):
    seq, margins = list(prompt), []
    for _ in range(n):
        top = forward(cfg, w, seq)[-1].topk(2)
        seq.append(int(top.indices[0]))
        margins.append(float(top.values[0] - top.values[1]))
    return seq[len(prompt):], margins
