"""Plain, slow restatement of the Kikurax layers for the tests: one function per mechanism, whole sequences at once
(no cache, no pages, no carried state), float64. Nothing here is shared with the product path; weights are the
checkpoint-named tensors."""

import math

import torch


# ---------------------------------------------------------------------------------- configurations
def rotary(base=1000.0, dims=16, factor=4.0, low=1.0, high=3.0, original=40):
    rot = {"base": base, "dims": dims}
    if factor:
        rot["scaling"] = {"factor": factor, "low": low, "high": high, "original": original}
    return rot


def attention(heads=4, kv_heads=2, dim=24, vdim=16, scale=0.3, softcap=8.0, v_mix=True, rot=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
                      "v_mix": v_mix, "rot": rot or rotary()}}


def left(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.25, coef=0.4, every=16):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
            "q_temp": {"coef": coef, "every": every}}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(a=None, b=None, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": a or left(), "right": b or delta()}}


def mamba2(heads=4, groups=2, state=16, vdim=24, conv=4, norm_groups=2, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv,
                                                    "norm_groups": norm_groups}}


def moe(ff=24, experts=6, top=2, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def random_config(layers, vocab=83, width=48, eps=1e-5, groups=3, scale=5.0):
    return {"architecture": "Kikurax", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
            "embedding": {"scale": scale}, "layers": layers}


# ---------------------------------------------------------------------------------- weights
def random_weights(cfg, seed=0, rank_a=10, rank_g=6):
    """bf16 tensors whose parts all matter: biases of either sign, decays from a token to hundreds, gates that open and
    close, mixing factors away from 0 and 1."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0):
        return (torch.randn(*shape, generator=g) * s).bfloat16()

    def lin(n, k, s=1.0):
        return rnd(n, k, s=s / math.sqrt(k))

    def near_one(n, s=0.2):
        return (1 + s * torch.randn(n, generator=g)).bfloat16()

    W, w = cfg["width"], {}
    w["embed"] = rnd(cfg["vocab"], W, s=1.0 / cfg["embedding"]["scale"])
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        q = p + "mix."
        w[p + "norm1"] = near_one(W)
        if layer["type"] == "attention":
            for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                w[q + n], w[q + n + ".b"] = lin(rows, W), rnd(rows, s=0.3)
            w[q + "temp"] = near_one(m["heads"], 0.4)
            if m.get("v_mix"):
                w[q + "vmix"] = torch.tensor(0.2 + 0.6 * float(torch.rand(1, generator=g))).bfloat16()
            w[q + "o"] = lin(W, m["heads"] * m["vdim"], 1.5)
        elif layer["type"] == "mamba2":
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            w[q + "in"] = lin(2 * inner + 2 * gn + m["heads"], W)
            w[q + "conv"], w[q + "conv.b"] = rnd(inner + 2 * gn, m["conv"], s=0.7), rnd(inner + 2 * gn, s=0.3)
            w[q + "dt_bias"], w[q + "A_log"] = rnd(m["heads"]) - 1, rnd(m["heads"], s=0.8) - 1
            w[q + "D"], w[q + "norm"], w[q + "o"] = near_one(m["heads"], 0.5), near_one(inner), lin(W, inner, 1.5)
        else:
            a, b, r = m["left"], m["right"], q + "right."
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"]),
                            ("g", a["heads"] * a["vdim"])):
                w[q + "left." + n] = lin(rows, W, 1.5)
            w[q + "left.pb"], w[q + "left.o"] = rnd(a["heads"]) - 2, lin(W, a["heads"] * a["vdim"])
            out = b["heads"] * b["vdim"]
            for n, rows in (("q", b["kv_heads"] * b["dim"]), ("k", b["kv_heads"] * b["dim"]), ("v", out)):
                w[r + n], w[r + n + ".conv"] = lin(rows, W), rnd(rows, b["conv"], s=0.7)
            w[r + "b"], w[r + "A_log"] = lin(b["heads"], W, 1.5), rnd(b["heads"], s=0.7) - 1
            w[r + "a1"], w[r + "a2"] = lin(rank_a, W), lin(b["heads"] * b["dim"], rank_a, 1.5)
            w[r + "dt_bias"] = rnd(b["heads"] * b["dim"], s=1.5) - 2
            w[r + "g1"], w[r + "g2"], w[r + "norm"] = lin(rank_g, W), lin(out, rank_g, 1.5), near_one(b["vdim"])
            w[r + "o"] = lin(W, out)
            w[q + "left.out"], w[q + "right.out"] = near_one(W), near_one(W)
        mlp, q = layer["mlp"], p + "mlp."
        if mlp is None:
            continue
        w[p + "norm2"] = near_one(W)
        w[q + "router"], w[q + "router.b"] = lin(mlp["router"]["experts"], W, 2.0), rnd(mlp["router"]["experts"])
        for e in range(mlp["router"]["experts"]):
            ff = mlp["expert"]["ff"]
            w[q + f"e{e}.gate"], w[q + f"e{e}.up"], w[q + f"e{e}.down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff)
    w["final.norm"] = near_one(W)
    return w


# ---------------------------------------------------------------------------------- elementary
def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log(1 + torch.exp(-z.abs())) + z.clamp_min(0)


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x, w, eps, groups):
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return over_rms(parts, eps).reshape(x.shape) * w.double()


def heads_of(x, n, d):
    """[T, n * d] -> [n, T, d]"""
    return x.reshape(x.shape[0], n, d).transpose(0, 1)


def short_conv(x, taps, bias=None):
    """x [T, C], taps [C, n]: the last tap belongs to the token itself; zeros before the start."""
    n = taps.shape[1]
    full = torch.cat([x.new_zeros(n - 1, x.shape[1]), x], 0)
    y = sum(full[j:j + x.shape[0]] * taps[:, j].double() for j in range(n))
    return silu(y if bias is None else y + bias.double())


# ---------------------------------------------------------------------------------- positions
def frequencies(rot):
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave, o = 2 * math.pi / f, s["original"]
            if wave > o / s["low"]:
                f = f / s["factor"]
            elif wave >= o / s["high"]:
                t = (o / wave - s["low"]) / (s["high"] - s["low"])
                f = (1 - t) * f / s["factor"] + t * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate(x, rot):
    """x [n, T, d]"""
    d = rot["dims"]
    a = torch.arange(x.shape[1], dtype=torch.float64)[:, None] * frequencies(rot)
    u, v = x[..., :d // 2], x[..., d // 2:d]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., d:]], -1)


def query_temperature(n, coef, every):
    return torch.tensor([1 + coef * math.log((p + 1) // every + 1) for p in range(n)], dtype=torch.float64)


# ---------------------------------------------------------------------------------- attention
def softcap(s, cap):
    return cap * torch.tanh(s / cap)


def sink_weights(s):
    """softmax over the keys of the past with one more term, e^0, in the denominator; s [T, T]."""
    e = torch.exp(s).tril()
    return e / (1 + e.sum(-1, keepdim=True))


def sigmoid_weights(s, bias):
    return sigmoid(s + bias).tril()


def attention_mixer(m, w, p, h, eps, first):
    """``first``: values of the first layer that mixes them, or None in that layer. Returns (output, own values)."""
    H, G = m["heads"], m["kv_heads"]

    def f(n):
        return w[p + n].double()

    q, k, v = (h @ f(n).T + f(n + ".b") for n in "qkv")
    own = v
    if m.get("v_mix") and first is not None:
        v = (1 - f("vmix")) * v + f("vmix") * first
    q = over_rms(rotate(heads_of(q, H, m["dim"]), m["rot"]), eps)
    k = over_rms(rotate(heads_of(k, G, m["dim"]), m["rot"]), eps)
    v = heads_of(v, G, m["vdim"])
    out = []
    for i in range(H):
        s = softcap(q[i] @ k[i // (H // G)].T * m["scale"] * f("temp")[i], m["softcap"])
        out.append(sink_weights(s) @ v[i // (H // G)])
    return torch.cat(out, -1) @ f("o").T, own


def left_mixer(m, w, p, h, eps):
    H, G = m["heads"], m["kv_heads"]

    def f(n):
        return w[p + n].double()

    q, k = over_rms(heads_of(h @ f("q").T, H, m["dim"]), eps), over_rms(heads_of(h @ f("k").T, G, m["dim"]), eps)
    v = heads_of(h @ f("v").T, G, m["vdim"])
    if m.get("q_temp"):
        q = q * query_temperature(h.shape[0], **m["q_temp"])[None, :, None]
    out = [sigmoid_weights(q[i] @ k[i // (H // G)].T * m["scale"], f("pb")[i]) @ v[i // (H // G)] for i in range(H)]
    return (torch.cat(out, -1) * sigmoid(h @ f("g").T)) @ f("o").T


# ---------------------------------------------------------------------------------- recurrences
def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, log_decay):
    """One head: q, k, log_decay [T, dk], v [T, dv], beta [T]."""
    S, out = q.new_zeros(q.shape[1], v.shape[1]), []
    for t in range(q.shape[0]):
        S = torch.exp(log_decay[t])[:, None] * S
        S = S + torch.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out.append(S.T @ q[t])
    return torch.stack(out)


def delta_mixer(m, w, p, h, eps):
    H, G, d = m["heads"], m["kv_heads"], m["dim"]

    def f(n):
        return w[p + n].double()

    q, k, v = (short_conv(h @ f(n).T, w[p + n + ".conv"]) for n in "qkv")
    q, k, v = unit(heads_of(q, G, d)) / math.sqrt(d), unit(heads_of(k, G, d)), heads_of(v, H, m["vdim"])
    beta = sigmoid(h @ f("b").T)
    dt = heads_of(softplus(h @ f("a1").T @ f("a2").T + f("dt_bias")), H, d)
    out = [over_rms(delta_rule(q[i // (H // G)], k[i // (H // G)], v[i], beta[:, i], -torch.exp(f("A_log")[i]) * dt[i]), eps)
           * f("norm") for i in range(H)]
    return (torch.cat(out, -1) * sigmoid(h @ f("g1").T @ f("g2").T)) @ f("o").T


def state_space(x, B, C, dt, a, D):
    """One head: x [T, dv], B and C [T, n], dt [T]."""
    S, out = x.new_zeros(B.shape[1], x.shape[1]), []
    for t in range(x.shape[0]):
        S = torch.exp(-a * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        out.append(S.T @ C[t] + D * x[t])
    return torch.stack(out)


def mamba2_mixer(m, w, p, h, eps):
    H, G, N, d = m["heads"], m["groups"], m["state"], m["vdim"]

    def f(n):
        return w[p + n].double()

    z, xbc, dt = (h @ f("in").T).split([H * d, H * d + 2 * G * N, H], -1)
    x, B, C = short_conv(xbc, w[p + "conv"], w[p + "conv.b"]).split([H * d, G * N, G * N], -1)
    x, B, C, dt = heads_of(x, H, d), heads_of(B, G, N), heads_of(C, G, N), softplus(dt + f("dt_bias"))
    y = torch.cat([state_space(x[i], B[i // (H // G)], C[i // (H // G)], dt[:, i], torch.exp(f("A_log")[i]), f("D")[i])
                   for i in range(H)], -1)
    return grouped_norm(y * silu(z), f("norm"), eps, m["norm_groups"]) @ f("o").T


# ---------------------------------------------------------------------------------- feed-forward
def expert(x, w, p, limit):
    g = (x @ w[p + "gate"].double().T).clamp_max(limit)
    u = (x @ w[p + "up"].double().T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].double().T


def routed(mlp, w, p, h, record=None):
    z, out = h @ w[p + "router"].double().T + w[p + "router.b"].double(), torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = sorted(range(z.shape[1]), key=lambda e: -float(z[t, e]))[:mlp["router"]["top"]]
        if record is not None:
            record.append(ids)
        e = torch.exp(z[t][ids] - z[t][ids].max())
        for i, share in zip(ids, e / e.sum()):
            out[t] += share * expert(h[t:t + 1], w, p + f"e{i}.", mlp["expert"]["limit"])[0]
    return out


# ---------------------------------------------------------------------------------- the model
def run_layer(cfg, w, i, x, first):
    """One layer; returns the residual and the values that later layers mix in."""
    layer, p, eps, groups = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"], cfg["norm"]["groups"]
    m, h = layer["mixer"], grouped_norm(x, w[p + "norm1"], eps, groups)
    p += "mix."
    if layer["type"] == "attention":
        y, own = attention_mixer(m, w, p, h, eps, first)
        if m.get("v_mix") and first is None:
            first = own
    elif layer["type"] == "mamba2":
        y = mamba2_mixer(m, w, p, h, eps)
    else:
        y = (over_rms(left_mixer(m["left"], w, p + "left.", h, eps), eps) * w[p + "left.out"].double() +
             over_rms(delta_mixer(m["right"], w, p + "right.", h, eps), eps) * w[p + "right.out"].double()) / 2
    x = x + y
    if layer["mlp"] is not None:
        x = x + routed(layer["mlp"], w, f"l{i}.mlp.", grouped_norm(x, w[f"l{i}.norm2"], eps, groups))
    return x, first


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] (float64); ``layers_out`` collects the residual after every layer."""
    x, first = w["embed"][torch.tensor(tokens)].double() * cfg["embedding"]["scale"], None
    for i in range(len(cfg["layers"])):
        x, first = run_layer(cfg, w, i, x, first)
        if layers_out is not None:
            layers_out.append(x)
    return grouped_norm(x, w["final.norm"], cfg["norm"]["eps"], cfg["norm"]["groups"]) @ w["embed"].double().T


def greedy(cfg, w, prompt, n):
    seq, margins = list(prompt), []
    for _ in range(n):
        top = forward(cfg, w, seq)[-1].topk(2)
        seq.append(int(top.indices[0]))
        margins.append(float(top.values[0] - top.values[1]))
    return seq[len(prompt):], margins
