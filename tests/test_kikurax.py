"""Kikurax through the framework's own engine against the plain restatement in ``helpers/kikurax_oracle.py``, on CPU (fp32)
and on a B200 (fp32 and bf16): whole prompts, decoding, portions, mixed batches, pages and state slots used again, which
tokens a position can see, greedy generation through the scheduler, pipeline stages, refit, loading and the trace runner."""

import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from helpers import kikurax_oracle as oracle
from helpers.kikurax_oracle import attention, delta, left, mamba2, moe, parallel, rotary
from parallax_b200.engine.engine import Engine
from parallax_b200.engine.request import Request, SamplingParams
from parallax_b200.loader.shard_loader import ShardLoader
from parallax_b200.models.config import config_from_hf, named_config

# layers that differ in everything; values mixed over layers with other mixers in between; feed-forwards or none
MIXED = oracle.random_config([
    mamba2(3, 1, 24, 16, norm_groups=3, mlp=moe()),
    attention(6, 2, 24, 16, mlp=moe(experts=5, top=3)),
    parallel(mlp=moe()),
    attention(2, 2, 32, 16, scale=0.2, softcap=3.0, rot=rotary(50.0, 8, 8.0, 1.0, 4.0, 30), mlp=None),
    parallel(left(6, 3, 16, 56, 0.4, 0.7, 5), delta(3, 3, 8, 40, conv=2), mlp=moe(top=1, limit=0.7)),
    attention(4, 1, 16, 48, v_mix=False, rot=rotary(300.0, 16, None), mlp=moe()),
    attention(8, 2, 8, 16, softcap=20.0, rot=rotary(20.0, 4, 2.0, 1.5, 2.5, 100), mlp=None)])
# sizes that no vector or tile width divides, one or five taps, wide eps, one key head
ODD = oracle.random_config([
    parallel(left(6, 3, 7, 5, 0.5, 1.3, 7), delta(6, 2, 9, 7, conv=5), mlp=moe(ff=11, experts=5, top=3)),
    mamba2(3, 3, 5, 7, conv=1, norm_groups=1, mlp=moe(ff=33, experts=3, top=3)),
    attention(3, 1, 11, 7, scale=0.6, rot=rotary(77.0, 6), mlp=None),
    attention(6, 1, 5, 7, scale=0.7, rot=rotary(77.0, 2), mlp=moe(ff=9, experts=7, top=2)),
    mamba2(6, 2, 3, 5, conv=3, norm_groups=5, mlp=None),
    parallel(left(1, 1, 3, 3, 0.5, 0.2, 1), delta(1, 1, 3, 3, conv=1), mlp=None)], vocab=37, width=30, eps=1e-3, groups=5, scale=3.0)
# equal sizes everywhere, one part of the norm, one expert per token, one head per group, factors of one
EQUAL = oracle.random_config([
    parallel(left(2, 2, 32, 32, 0.2, 0.3, 64), delta(2, 2, 32, 32), mlp=moe(ff=64, experts=4, top=1, limit=1.0)),
    attention(2, 2, 32, 32, softcap=1.0, rot=rotary(1000.0, 32, 1.0, 1.0, 2.0, 64), mlp=moe(ff=64, experts=1, top=1)),
    mamba2(2, 2, 32, 32, norm_groups=1, mlp=moe(ff=64, experts=4, top=4))], vocab=64, width=64, groups=1, scale=1.0)
# tensor-core widths: 64 and 128 columns per head, states of several slices, heads that share q and k, many query heads
WIDE = oracle.random_config([
    parallel(left(8, 2, 96, 128, 0.1, 0.4, 20), delta(4, 2, 64, 96), mlp=moe(ff=96, experts=10, top=4)),
    attention(8, 2, 64, 48, scale=0.2, softcap=15.0, rot=rotary(1000.0, 64), mlp=moe(ff=72, experts=6, top=2)),
    mamba2(6, 2, 64, 40, norm_groups=4, mlp=moe(ff=64)),
    parallel(left(4, 4, 48, 64, 0.2, 0.4, 30), delta(2, 1, 128, 128, conv=3), mlp=None),
    attention(4, 2, 128, 48, scale=0.12, softcap=30.0, rot=rotary(1000.0, 64), mlp=None),
    mamba2(2, 1, 128, 64, norm_groups=1, mlp=None),
    attention(34, 2, 16, 24, scale=0.3, v_mix=False, rot=rotary(1000.0, 16), mlp=None)], vocab=200, width=128, groups=2)
CONFIGS = {"mixed": MIXED, "odd": ODD, "equal": EQUAL, "wide": WIDE}
SPREAD = {"odd": 1.6, "equal": 1.6}      # narrow models: rounding to bf16 shows more
_weights, _logits = {}, {}

GPU = pytest.mark.gpu
TARGETS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda:0", torch.float32), id="gpu-fp32", marks=GPU),
           pytest.param(("cuda:0", torch.bfloat16), id="gpu-bf16", marks=GPU)]


def weights(name):
    if name not in _weights:
        _weights[name] = oracle.random_weights(CONFIGS[name], seed=len(name))
    return _weights[name]


def tokens(name, n, seed=0):
    g = torch.Generator().manual_seed(100 + seed)
    return torch.randint(0, CONFIGS[name]["vocab"], (400,), generator=g).tolist()[:n]


def want_logits(name, n, seed=0):
    """Oracle logits of a random sequence (causal: also those of its prefixes)."""
    key = (name, seed)
    if key not in _logits or _logits[key].shape[0] < n:
        _logits[key] = oracle.forward(CONFIGS[name], weights(name), tokens(name, n, seed))
    return _logits[key][:n]


def engine(cfg, target, w=None, **kw):
    dev, dt = target
    args = dict(page_size=16, num_blocks=40, max_batch_size=4, max_num_tokens_per_batch=512, max_total_length=400,
                enable_prefix_cache=False, max_requests=4)
    args.update(kw)
    if isinstance(cfg, str):
        cfg, w = CONFIGS[cfg], weights(cfg)
    return Engine(config_from_hf(cfg), device=dev, dtype=dt, weights=w, **args)


def errors(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std(-1)


def close(got, want, target, what="", spread=1.0):
    """In bf16 a close call of a router may fall the other way: a few positions may be off, the bulk may not."""
    err = errors(got, want)
    if target[1] == torch.float32:
        assert float(err.max()) < 5e-5, (what, float(err.max()))
    else:
        assert float(err.median()) < 4e-2 * spread and float(err.quantile(0.8)) < 1e-1 * spread and float(err.max()) < 1.2, \
            (what, [float(err.quantile(q)) for q in (0.5, 0.8, 1.0)])


# ---------------------------------------------------------------------------------- whole prompts and layers
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(name, target):
    eng = engine(name, target)
    for n in (1, 2, 17, 64, 65, 113):
        got = eng.feed([("r", tokens(name, n), range(n))])
        close(got, want_logits(name, 113)[:n], target, n, SPREAD.get(name, 1.0))
        eng.release_fed("r")
    assert eng.cache.num_free_blocks() == 40


@pytest.mark.parametrize("target", TARGETS)
def test_residual_after_every_stage(target):
    """Stages are cut where no layer mixes in the values of an earlier one."""
    cfg, n = oracle.random_config([parallel(mlp=moe()), mamba2(mlp=moe()), attention(mlp=moe()), attention(mlp=None)]), 60
    w, ref = oracle.random_weights(cfg, seed=8), []
    seq = tokens("mixed", n)
    want = oracle.forward(cfg, w, seq, ref)
    eng = engine(cfg, target, w, stage_layers=[(0, 1), (1, 2), (2, 4)])
    seen = []
    eng.wire_hook = lambda h: (seen.append(h.clone()), h)[1]      # hidden states between pipeline stages
    close(eng.feed([("r", seq, range(n))]), want, target)
    assert len(ref) == 4 and len(seen) == 2 and all(h.dtype == torch.float32 for h in seen)
    for h, x in zip(seen, ref):
        err = (h.double().cpu() - x).norm(dim=-1) / x.norm(dim=-1)
        assert float(err.quantile(0.8)) < (2e-5 if target[1] == torch.float32 else 3e-2)


# ---------------------------------------------------------------------------------- decoding and portions
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_decoding_equals_the_prompt(name, target):
    """Token by token from the first token on, over page borders and changes of the query temperature."""
    n = 118
    eng, seq = engine(name, target), tokens(name, n)
    got = torch.cat([eng.feed([("r", [t], [0])]) for t in seq])
    close(got, want_logits(name, n), target, "", SPREAD.get(name, 1.0))


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("cut", [(2,), (3, 1, 5), (16,), (15, 17, 1, 1, 31), (64, 2), (63, 3)])
def test_portions_of_any_size(name, target, cut):
    n = 110
    eng, seq = engine(name, target), tokens(name, n)
    got, at, k = [], 0, 0
    while at < n:
        m = min(cut[k % len(cut)], n - at)
        got.append(eng.feed([("r", seq[at:at + m], range(m))]))
        at, k = at + m, k + 1
    close(torch.cat(got), want_logits(name, n), target, cut, SPREAD.get(name, 1.0))


@pytest.mark.parametrize("target", TARGETS)
def test_long_decoding(target):
    name, n = "mixed", 330
    eng, seq = engine(name, target), tokens(name, n)
    eng.feed([("r", seq[:3], [])])
    got = torch.cat([eng.feed([("r", [t], [0])]) for t in seq[3:]])
    close(got, want_logits(name, n)[3:], target)


@pytest.mark.parametrize("target", [TARGETS[1], TARGETS[2]])
def test_portions_agree_with_the_whole_prompt_on_the_gpu(target):
    """The same weights and kernels: only rounding may differ, so routers fall the same way almost everywhere."""
    name, n = "wide", 230
    eng, seq = engine(name, target), tokens(name, n)
    whole = eng.feed([("a", seq, range(n))])
    parts = torch.cat([eng.feed([("b", seq[i:i + 37], range(len(seq[i:i + 37])))]) for i in range(0, n, 37)])
    err = errors(parts, whole)
    assert float(err.quantile(0.8)) < (1e-5 if target[1] == torch.float32 else 3e-2)


# ---------------------------------------------------------------------------------- what a position can see
SIGHT = {  # one layer each: sizes of the tensor-core kernels and others
    "attention-24": attention(2, 1, 24, 16, rot=rotary(1000.0, 8)),
    "attention-64": attention(4, 2, 64, 48, scale=0.1, rot=rotary(1000.0, 16)),
    "attention-128": attention(4, 1, 128, 128, scale=0.06, rot=rotary(1000.0, 64)),
    "sigmoid-and-delta": parallel(left(2, 1, 16, 16, 0.2), delta(1, 1, 32, 32)),
    "state-space": mamba2(2, 1, 32, 32, norm_groups=1),
}


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("which", sorted(SIGHT))
def test_a_changed_token_shows_exactly_where_it_is_seen(which, target):
    """Another token at one place changes the logits of it and of every later position, and not a bit of any earlier one:
    first tokens, page borders, in prompts, portions and decoding."""
    cfg = oracle.random_config([SIGHT[which]], vocab=50, width=64, groups=2)
    w = oracle.random_weights(cfg, seed=3)
    for name in w:
        if name.endswith("dt_bias"):
            w[name] = torch.full_like(w[name], -5.0)      # a memory that keeps what it has seen
        if name.endswith("A_log"):
            w[name] = torch.full_like(w[name], -2.0)
    eng, n = engine(cfg, target, w), 210
    seq = torch.randint(0, 50, (n,), generator=torch.Generator().manual_seed(1)).tolist()

    def run(s):
        """A prompt, a portion of two, a longer one, then single tokens."""
        cuts, out, at = [130, 2, 40] + [1] * (n - 172), [], 0
        for m in cuts:
            out.append(eng.feed([("r", s[at:at + m], range(m))]).cpu())
            at += m
        eng.release_fed("r")
        return torch.cat(out)

    base = run(seq)
    for j in (0, 1, 15, 16, 17, 63, 64, 129, 130, 131, 171, 172, n - 2, n - 1):
        other = run(seq[:j] + [(seq[j] + 7) % 50] + seq[j + 1:])
        changed = (other != base).any(-1)
        assert not bool(changed[:j].any()), j
        if target[1] == torch.bfloat16:       # a key with next to no weight may leave every rounded logit alone
            assert bool(changed[j:][-40:].any()) and bool(changed[j]), j
        else:
            assert bool(changed[j:].all()), (j, (~changed[j:]).nonzero().flatten().tolist())


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("what", ["sink", "temp", "softcap", "vmix", "bias", "q_temp", "pb", "conv", "decay", "skip", "router", "limit",
                                  "stretch", "key"])
def test_small_print_matters(what, target):
    """Weights and constants that only one mechanism reads, made large: leaving it out would show far beyond rounding."""
    n = 70
    cfg = json.loads(json.dumps(oracle.random_config([parallel(mlp=moe()), mamba2(mlp=moe()), attention(mlp=moe()),
                                                      attention(mlp=None)])))
    w, seq, spread = oracle.random_weights(cfg, seed=21), tokens("mixed", n), 1.0
    plain = oracle.forward(cfg, w, seq)
    m = [e["mixer"] for e in cfg["layers"]]
    if what == "sink":          # scores far below 0: nearly all of the weight goes to the added one
        w["l2.mix.q.b"], w["l2.mix.k.b"] = 6 + w["l2.mix.q.b"], w["l2.mix.k.b"] - 6
        m[2]["softcap"] = 3.0
    elif what == "temp":
        w["l2.mix.temp"], w["l3.mix.temp"] = torch.tensor([4.0, -3.0, 0.0, 2.0]).bfloat16(), -w["l3.mix.temp"]
    elif what == "softcap":
        m[2].update(softcap=0.4, scale=2.0)
    elif what == "vmix":
        w["l3.mix.vmix"] = torch.tensor(-3.0).bfloat16()
    elif what == "bias":
        w["l2.mix.v.b"] = w["l2.mix.v.b"] + 4
    elif what == "q_temp":
        m[0]["left"]["q_temp"] = {"coef": 3.0, "every": 2}
    elif what == "pb":
        w["l0.mix.left.pb"] = torch.tensor([5.0, -9.0, 0.0, -1.0]).bfloat16()
    elif what == "conv":
        w["l1.mix.conv"], w["l0.mix.right.v.conv"] = w["l1.mix.conv"].flip(1) * 2, w["l0.mix.right.v.conv"].flip(1) * 2
        w["l1.mix.conv.b"] = w["l1.mix.conv.b"] + 1
    elif what == "decay":
        w["l0.mix.right.A_log"] = torch.tensor([3.0, -6.0, 1.0, 2.0]).bfloat16()
        w["l1.mix.A_log"], w["l1.mix.dt_bias"] = torch.tensor([4.0, -6.0, 0.0, 2.0]).bfloat16(), 3 + w["l1.mix.dt_bias"]
    elif what == "skip":
        w["l1.mix.D"] = torch.tensor([6.0, -5.0, 0.0, 3.0]).bfloat16()
    elif what == "router":
        w["l0.mlp.router.b"] = torch.tensor([0.0, 30.0, 0.0, 30.0, 0.0, -5.0]).bfloat16()
    elif what == "limit":
        cfg["layers"][0]["mlp"]["expert"]["limit"] = 0.05
    elif what == "stretch":
        m[2]["rot"]["scaling"] = {"factor": 30.0, "low": 0.5, "high": 20.0, "original": 60}
    else:                       # one far key among all others
        w["embed"] = w["embed"].clone()
        seq = [5 if t == 7 else t for t in seq]
        seq[3] = 7
        w["embed"][7] = 30 * w["embed"][7]
    want = oracle.forward(cfg, w, seq)
    got = engine(cfg, target, w).feed([("r", seq, range(n))])
    close(got, want, target, what, spread)
    if what != "key":
        assert float(errors(plain, want).median()) > 0.1


# ---------------------------------------------------------------------------------- batches, pages, slots
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_requests_in_one_batch(name, target):
    """Portions beside decoded tokens, requests left out of steps; pages and state slots change hands, and whatever earlier
    owners left in them must not show."""
    eng = engine(name, target, num_blocks=26)
    for lc in eng.stages[0].pool.caches():
        for t in (lc.k, lc.v, lc.rec_state, lc.conv_state):
            if t is not None:
                t.fill_(37.0)                 # what it held before it was handed out
    plan = [  # per step: (request, seed, tokens)
        [("a", 1, 40), ("b", 2, 1), ("c", 3, 2)], [("b", 2, 1), ("a", 1, 1), ("d", 4, 90)], [("c", 3, 33), ("a", 1, 1)],
        [("d", 4, 1), ("c", 3, 1), ("b", 2, 50), ("a", 1, 7)], [("a", 1, 60), ("d", 4, 1)]]
    for round_ in range(3):
        at = {}
        for step in plan:
            entries, refs = [], []
            for rid, seed, m in step:
                lo = at.get(rid, 0)
                entries.append((rid, tokens(name, 118, seed)[lo:lo + m], range(m)))
                refs.append(want_logits(name, 118, seed)[lo:lo + m])
                at[rid] = lo + m
            close(eng.feed(entries), torch.cat(refs), target, (round_, step))
        for rid in ("b", "d", "a", "c"):
            eng.release_fed(rid)
        assert eng.cache.num_free_blocks() == 26


# ---------------------------------------------------------------------------------- generation through the scheduler
def generate(eng, prompts, n):
    reqs = [Request(input_ids=p, sampling_params=SamplingParams(max_new_tokens=n, temperature=0.0, ignore_eos=True),
                    max_total_length=400) for p in prompts]
    for r in reqs:
        eng.add_request(r)
    while eng.has_work():
        eng.step()
    return [r.output_ids for r in reqs], sum(r.num_cached_tokens for r in reqs)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("kw", [dict(), dict(chunked_prefill_size=7), dict(enable_prefix_cache=True, chunked_prefill_size=16),
                                dict(stage_layers=[(0, 1), (1, 7)])], ids=["plain", "slices", "prefix-cache", "stages"])
def test_greedy_generation(target, kw):
    """More requests than the batch holds; with the prefix cache, requests resume from snapshots of the states and of the
    convolutions' inputs at a block's end."""
    name, n_new = "mixed", 7
    kw = dict(dict(max_requests=None, max_num_tokens_per_batch=60), **kw)
    eng = engine(name, target, **kw)
    base = tokens(name, 70, 9)
    prompts = [base[:33], tokens(name, 1, 5), base[:48], tokens(name, 27, 6), base[:64], base[:32] + tokens(name, 3, 7)]
    outs, _ = generate(eng, prompts, n_new)
    again, cached = generate(eng, prompts, n_new)
    assert (cached >= 32 * 3) == bool(kw.get("enable_prefix_cache"))
    for p, got, got2 in zip(prompts, outs, again):
        want, margins = oracle.greedy(CONFIGS[name], weights(name), p, n_new)
        for i in range(n_new):
            if target[1] == torch.bfloat16 and margins[i] < 0.5:      # a near tie may fall either way in bf16
                break
            assert got[i] == want[i] == got2[i], (len(p), i, margins[i])


@pytest.mark.parametrize("target", TARGETS)
def test_sampled_requests_and_penalties_run(target):
    eng = engine("mixed", target, max_requests=None)
    sp = SamplingParams(max_new_tokens=5, temperature=0.8, top_k=5, repetition_penalty=1.2, ignore_eos=True)
    outs = eng.generate([tokens("mixed", 20), tokens("mixed", 3)], sp)
    assert all(len(o) == 5 and all(0 <= t < CONFIGS["mixed"]["vocab"] for t in o) for o in outs)


@pytest.mark.parametrize("target", TARGETS)
def test_routed_experts_are_recorded(target):
    """The record of the experts every token went to (biased logits decide)."""
    cfg = oracle.random_config([mamba2(mlp=moe(experts=5, top=2))])
    w = oracle.random_weights(cfg, seed=4)
    w["l0.mlp.router.b"] = torch.tensor([0.0, 50.0, 0.0, 0.0, 40.0]).bfloat16()
    eng = engine(cfg, target, w, max_requests=None, return_routed_experts=True)
    req = Request(input_ids=tokens("mixed", 9), sampling_params=SamplingParams(max_new_tokens=3, temperature=0.0, ignore_eos=True),
                  max_total_length=40)
    eng.add_request(req)
    while eng.has_work():
        eng.step()
    ids = torch.as_tensor(req.routed_experts).reshape(-1, 2)
    assert ids.shape[0] >= 9 and bool((ids == torch.tensor([1, 4])).all())


# ---------------------------------------------------------------------------------- configuration, loading, refit
def write_model(tmp_path, name):
    from safetensors.torch import save_file

    (tmp_path / "config.json").write_text(json.dumps(CONFIGS[name]))
    save_file(weights(name), str(tmp_path / "model.safetensors"))
    return str(tmp_path)


def test_loader_selects_a_stages_tensors(tmp_path):
    from parallax_b200.loader.filter import filter_weight_files

    path = write_model(tmp_path, "mixed")
    a, b = set(ShardLoader(path, 0, 3).load_weights()), set(ShardLoader(path, 3, 7).load_weights())
    assert {"embed", "l0.mix.in", "l1.mix.q.b", "l2.mix.right.a2"} <= a and not any(k.startswith("l3.") for k in a)
    assert {"embed", "final.norm", "l3.mix.vmix", "l5.mlp.e4.down"} <= b and "final.norm" not in a
    assert a | b == set(weights("mixed")) and a & b == {"embed"}
    assert "embed" not in set(ShardLoader(path, 1, 3).load_weights())
    files = {"embed": "x.safetensors", "l0.norm1": "y.safetensors", "l6.norm1": "z.safetensors"}
    (tmp_path / "model.safetensors.index.json").write_text(json.dumps({"weight_map": files}))
    assert filter_weight_files(path, sorted(files.values()), 6, 7, False, True) == ["x.safetensors", "z.safetensors"]


def edited(path, value):
    cfg = json.loads(json.dumps(MIXED))
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return cfg


def test_config_errors():
    for path, value, text in ((("layers", 0, "type"), "something_else", "something_else"),
                              (("layers", 0, "mlp", "kind"), "dense", "dense"),
                              (("layers", 1, "mixer", "kv_heads"), 4, "evenly"),
                              (("layers", 2, "mixer", "left", "kv_heads"), 3, "evenly"),
                              (("layers", 2, "mixer", "right", "kv_heads"), 3, "no delta rule"),
                              (("layers", 0, "mixer", "groups"), 2, "no state-space"),
                              (("layers", 0, "mixer", "norm_groups"), 5, "no state-space"),
                              (("layers", 1, "mixer", "rot", "dims"), 25, "rotary"),
                              (("layers", 1, "mixer", "rot", "scaling", "high"), 1.0, "stretches"),
                              (("layers", 3, "mixer", "vdim"), 24, "width of their value heads"),
                              (("norm", "groups"), 5, "equal parts"),
                              (("layers", 0, "mlp", "shared"), {"ff": 8}, "not part of"),
                              (("layers", 0, "mlp", "router", "top"), 7, "to choose from")):
        with pytest.raises(ValueError, match=text):
            config_from_hf(edited(path, value))
    cfg = config_from_hf(MIXED)
    assert [cfg.layer_kind(i) for i in range(7)] == ["linear", "attention", "attention", "attention", "attention", "attention", "attention"]
    assert cfg.linked_layers == [(1, 3), (1, 6)] and cfg.tie_word_embeddings and cfg.norm_groups == 3
    assert cfg.kv_dims(0) is None and cfg.kv_dims(1) == (2, 64) and cfg.has_linear_layers
    assert cfg.slot_dims(1) is None and cfg.slot_dims(4) == ((1, 24 + 24 + 120), (3, 8, 40))
    short = {k: v for k, v in weights("mixed").items() if k != "l4.mix.right.out"}
    with pytest.raises(KeyError, match="l4.mix.right.out"):
        Engine(cfg, device="cpu", num_blocks=8, weights=short)
    wrong = dict(weights("mixed"), **{"l2.mix.right.a1": torch.zeros(11, 48)})
    with pytest.raises(ValueError, match="do not fit together"):
        Engine(cfg, device="cpu", num_blocks=8, weights=wrong)
    wrong = dict(weights("mixed"), **{"l2.mix.right.a1": torch.zeros(10, 47)})
    with pytest.raises(ValueError, match="l2.mix.right.a1"):
        Engine(cfg, device="cpu", num_blocks=8, weights=wrong)
    with pytest.raises(ValueError, match="one pipeline stage"):
        Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), stage_layers=[(0, 2), (2, 7)])
    with pytest.raises(ValueError, match="quantised pages"):
        Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), kv_cache_dtype="fp8_e4m3")
    from parallax_b200.models.registry import build_stage

    with pytest.raises(ValueError, match="tensor parallelism"):
        build_stage(cfg, 0, 7, "cpu", torch.float32, tp_size=2)
    with pytest.raises(ValueError, match="expert parallelism"):
        build_stage(cfg, 0, 7, "cpu", torch.float32, ep_size=2)
    with pytest.raises(ValueError, match="LoRA"):
        Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), lora={"max_loaded": 1, "paths": {}})


def test_stretched_frequencies():
    from parallax_b200.models.rope import stretched_frequencies

    rot = rotary(1000.0, 48, 8.0, 1.0, 4.0, 200)
    plain = torch.tensor([1000.0 ** (-2 * i / 48) for i in range(24)], dtype=torch.float64)
    got = stretched_frequencies(plain, 8.0, 1.0, 4.0, 200.0)
    torch.testing.assert_close(got, oracle.frequencies(rot), rtol=1e-12, atol=0)
    assert bool((got == plain).any()) and bool((got == plain / 8).any()) and bool(((got < plain) & (got > plain / 8)).any())


def test_cluster_model_info_of_a_layer_list_config():
    from parallax_b200.backend.static_config import model_info_from_config

    info = model_info_from_config(MIXED, "x")
    assert (info.num_layers, info.hidden_dim, info.vocab_size, info.num_attention_heads) == (7, 48, 83, 8)
    assert info.num_local_experts == 6 and info.num_experts_per_tok == 3 and info.tie_embedding


def test_sizes_of_pages_and_slots():
    """A layer with two mixers has pages and a slot; slots hold the convolutions' inputs and the fp32 state."""
    from parallax_b200.cache.kv_pool import KVPool, bytes_per_block, bytes_per_linear_slot

    cfg = config_from_hf(MIXED)
    pool = KVPool(cfg, 0, 7, 7, 16, "cpu", torch.float32, num_linear_slots=3)
    per_token = 2 * 64 * (2 + 2 + 2 + 3 + 1 + 2)
    assert bytes_per_block(cfg, 0, 7, 16, 4) == 16 * 4 * per_token
    conv = 3 * (48 + 24 + 24) + 3 * (32 + 32 + 96) + 1 * (24 + 24 + 120)
    state = 3 * 24 * 16 + 4 * 16 * 24 + 3 * 8 * 40
    assert bytes_per_linear_slot(cfg, 0, 7, 4) == 4 * (conv + state) and bytes_per_linear_slot(cfg, 0, 7, 2) == 2 * conv + 4 * state
    assert 3 * bytes_per_linear_slot(cfg, 0, 7, 4) + 7 * bytes_per_block(cfg, 0, 7, 16, 4) == pool.nbytes()
    for t in pool._slot_tensors():
        t[1].fill_(5.0)
    pool.copy_slot(2, 1)
    pool.zero_slot(1)
    assert len(pool._slot_tensors()) == 6
    assert all(bool((t[2] == 5).all()) and bool((t[1] == 0).all()) for t in pool._slot_tensors())


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("stages", [None, [(0, 1), (1, 7)]])
def test_refit(target, stages):
    name, n = "mixed", 40
    eng = engine(name, target, stage_layers=stages)
    other = oracle.random_weights(CONFIGS[name], seed=77)
    eng.update_weights({k: v for k, v in other.items() if not k.startswith("l2.")})
    new = {k: (weights(name) if k.startswith("l2.") else other)[k] for k in other}
    close(eng.feed([("r", tokens(name, n), range(n))]), oracle.forward(CONFIGS[name], new, tokens(name, n)), target)
    eng.release_fed("r")
    eng.update_weights({k: v for k, v in weights(name).items() if k.startswith(("l3.", "l5."))})     # layers without the table
    new = {k: (weights(name) if k.startswith(("l2.", "l3.", "l5.")) else other)[k] for k in other}
    close(eng.feed([("r", tokens(name, n), range(n))]), oracle.forward(CONFIGS[name], new, tokens(name, n)), target)


@pytest.mark.parametrize("name", ["tiny-kikurax", "small-kikurax"])
def test_named_configs_build(name):
    eng = Engine(named_config(name), device="cpu", num_blocks=16, max_batch_size=2)
    assert len(eng.generate([[1, 2, 3]], SamplingParams(max_new_tokens=3, temperature=0.0))[0]) == 3


def test_offline_generation_command(tmp_path):
    from parallax_b200.generate import run

    res = run(write_model(tmp_path, "mixed"), "hello", max_tokens=4, device="cpu", out=lambda _line: None)
    assert res["generated_tokens"] == 4


# ---------------------------------------------------------------------------------- trace runner
@pytest.mark.parametrize("dtype", [pytest.param("float32", id="fp32"), pytest.param("bfloat16", id="bf16", marks=GPU)])
def test_trace_runner(tmp_path, dtype):
    import numpy as np

    name = "mixed"
    seq = tokens(name, 90)
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": seq[:30], "want": [0, 29]},
                                     {"id": "q", "tokens": seq[:2], "want": [1]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": seq[2:3], "want": []}], "end": ["q"]},
             {"step": 4, "entries": [{"id": "p", "tokens": seq[30:31], "want": [0]},
                                     {"id": "s", "tokens": seq[:64], "want": [63, 5]}], "end": ["p", "s"]},
             {"step": 5, "entries": [{"id": "p", "tokens": seq, "want": [89]}], "end": ["p"]}]
    model, out = tmp_path / "m", tmp_path / "o"
    model.mkdir()
    out.mkdir()
    runner = Path(__file__).resolve().parent.parent / "bin" / "trace_run"
    res = subprocess.run([sys.executable, str(runner), "--model", write_model(model, name), "--dtype", dtype, "--out", str(out),
                          "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                         text=True, timeout=300, env=dict(os.environ, OMP_NUM_THREADS="2"))
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 4", "done 5"]
    ref, V = want_logits(name, 90), CONFIGS[name]["vocab"]
    target = ("cpu", torch.float32 if dtype == "float32" else torch.bfloat16)
    rows, refs = [], []
    for step, places in ((0, [0, 29, 1]), (4, [30, 63, 5]), (5, [89])):
        rows.append(torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(places), V)))
        refs.append(ref[places])
    close(torch.cat(rows), torch.cat(refs), target)
    assert not (out / "1.f32").exists()
