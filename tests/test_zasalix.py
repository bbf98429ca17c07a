"""Zasalix through the framework's own engine against the plain restatement in ``helpers/zasalix_oracle.py``, on CPU (fp32)
and on a B200 (fp32 and bf16): whole prompts, decoding, portions, mixed batches, pages and state slots used again, which
tokens a position can see, greedy generation through the scheduler, pipeline stages, refit, loading and the trace runner."""

import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from helpers import zasalix_oracle as oracle
from helpers.zasalix_oracle import dense, latent, memory, mlstm, moe, parallel, windowed
from parallax_b200.engine.engine import Engine
from parallax_b200.engine.request import Request, SamplingParams
from parallax_b200.loader.shard_loader import ShardLoader
from parallax_b200.models.config import config_from_hf, named_config

# layers that differ in everything, a loop in the middle, every feed-forward behind every mixer, or none
MIXED = oracle.random_config([
    mlstm(3, 16, 8, mlp=dense(72)),
    parallel(windowed(6, 2, 24, 16, rot=16, scale=0.3, size=20, keep=5), memory(2, 24, 40), mlp=moe()),
    latent(mlp=moe(experts=5, top=3, shared=None)),
    parallel(windowed(2, 1, 40, 56, rot=8, base=50.0, scale=0.15, size=33, keep=17), memory(3, 8, 16), (-0.4, 1.2), mlp=None),
    latent(2, 24, 16, 20, 48, 40, base=50.0, scale=0.3, mlp=dense(40)),
    mlstm(1, 32, 48, mlp=moe(top=1))], loop=(1, 3, 2))
# sizes that no vector or tile width divides, an odd token input, three passes over the first two layers, wide eps
ODD = oracle.random_config([
    latent(3, 5, 6, 7, 9, 11, scale=0.5, mlp=moe(ff=11, experts=5, top=3, shared=13)),
    parallel(windowed(6, 3, 7, 5, rot=4, scale=0.5, size=7, keep=3), memory(3, 9, 7, cap=2.0), mlp=dense(33)),
    mlstm(1, 5, 3, cap=3.0, mlp=None)], vocab=37, width=30, eps=1e-3, side=7, loop=(0, 2, 3))
# equal sizes everywhere, factors and passes of one, one expert per token, nothing kept in front of the window
EQUAL = oracle.random_config([
    parallel(windowed(2, 2, 32, 32, rot=32, scale=0.2, size=32, keep=0), memory(2, 32, 32, cap=1.0), (1.0, 1.0),
             mlp=moe(ff=64, experts=4, top=1, shared=64)),
    latent(2, 32, 32, 32, 32, 32, scale=0.2, mlp=dense(64)), mlstm(2, 32, 32, cap=1.0, mlp=dense(64))], vocab=64, width=64, side=64,
    loop=(1, 3, 1))
# tensor-core widths: 64 and 128 columns per head, several slices of a memory, latents wider than a chunk, many heads
WIDE = oracle.random_config([
    parallel(windowed(8, 2, 48, 64, rot=32, scale=0.15, size=70, keep=9), memory(2, 64, 96), mlp=moe(ff=96, experts=10, top=4, shared=128)),
    latent(8, 64, 32, 64, 192, 128, scale=0.1, mlp=dense(256)),
    parallel(windowed(8, 2, 128, 96, rot=64, scale=0.09, size=40, keep=65), memory(1, 128, 128), mlp=dense(136)),
    latent(20, 16, 8, 24, 64, 64, mlp=None),
    parallel(windowed(34, 2, 16, 24, rot=16, scale=0.3, size=100, keep=20), memory(2, 48, 64), mlp=None)],
    vocab=200, width=128, side=32, loop=(2, 4, 2))
# no loop, no token input
PLAIN = oracle.random_config([latent(mlp=dense()), mlstm(mlp=moe())], side=0, loop=None)
CONFIGS = {"mixed": MIXED, "odd": ODD, "equal": EQUAL, "wide": WIDE, "plain": PLAIN}
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
        close(got, want_logits(name, 113)[:n], target, n)
        eng.release_fed("r")
    assert eng.cache.num_free_blocks() == 40


@pytest.mark.parametrize("target", TARGETS)
def test_residual_after_every_stage(target):
    """Stages may be cut anywhere behind the loop; every one reads the token ids for its layers' inputs."""
    name, n = "mixed", 60
    ref = []
    oracle.forward(CONFIGS[name], weights(name), tokens(name, n), ref)
    eng = engine(name, target, stage_layers=[(0, 3), (3, 4), (4, 6)])
    seen = []
    eng.wire_hook = lambda h: (seen.append(h.clone()), h)[1]      # hidden states between pipeline stages
    close(eng.feed([("r", tokens(name, n), range(n))]), want_logits(name, n), target)
    assert len(ref) == 8 and len(seen) == 2 and all(h.dtype == torch.float32 for h in seen)
    for h, x in zip(seen, (ref[4], ref[5])):
        err = (h.double().cpu() - x).norm(dim=-1) / x.norm(dim=-1)
        assert float(err.quantile(0.8)) < (2e-5 if target[1] == torch.float32 else 3e-2)


# ---------------------------------------------------------------------------------- decoding and portions
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_decoding_equals_the_prompt(name, target):
    """Token by token from the first token on, over page borders and window edges."""
    n = 118
    eng, seq = engine(name, target), tokens(name, n)
    got = torch.cat([eng.feed([("r", [t], [0])]) for t in seq])
    close(got, want_logits(name, n), target)


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
    close(torch.cat(got), want_logits(name, n), target, cut)


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
SIGHT = {  # one layer each, sizes of the tensor-core kernels and others; (layer, tokens seen by i)
    "window-24": (parallel(windowed(2, 1, 24, 16, rot=8, scale=0.2, size=20, keep=5), (0.8, 0.0)), 20, 5),
    "window-64": (parallel(windowed(4, 2, 48, 64, rot=16, scale=0.1, size=70, keep=9), (0.8, 0.0)), 70, 9),
    "window-128": (parallel(windowed(4, 1, 128, 128, rot=64, scale=0.06, size=64, keep=130), (0.8, 0.0)), 64, 130),
    "latent": (latent(2, 16, 8, 16, 32, 24, scale=0.1), None, 0),
    "memory": (mlstm(1, 32, 32), None, 0),
}
for _layer, _size, _keep in SIGHT.values():
    if _layer["type"] == "parallel":        # (factors of the two mixers: only the window is left)
        _layer["mixer"].update(right=memory(1, 8, 8), left_scale=0.8, right_scale=0.0)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("which", sorted(SIGHT))
def test_a_changed_token_shows_exactly_where_it_is_seen(which, target):
    """Another token at one place changes the logits of every position that sees it and not a bit of any other: just inside
    and outside the window, the kept first tokens and the next ones, page borders, in prompts, portions and decoding."""
    layer, size, keep = SIGHT[which]
    cfg = oracle.random_config([layer], vocab=50, width=64, side=0, loop=None)
    w = oracle.random_weights(cfg, seed=3)
    for name in w:
        if name.endswith("mix.f.b"):
            w[name] = torch.full_like(w[name], 9.0)       # a memory that keeps what it has seen
        if name.endswith("mix.f"):
            w[name] = w[name] * 0
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
    places = {0, 1, keep - 1, keep, keep + 1, 15, 16, 17, 129, 130, 131, 171, 172, n - 2, n - 1}
    if size:
        places |= {130 - size, 131 - size, 172 - size, 173 - size, n - 1 - size, n - size}
    for j in sorted(p for p in places if 0 <= p < n):
        other = run(seq[:j] + [(seq[j] + 7) % 50] + seq[j + 1:])
        changed = (other != base).any(-1)
        want = torch.tensor([oracle.seen(i, j, size, keep) for i in range(n)])
        if target[1] == torch.bfloat16:       # a key with next to no weight may leave every rounded logit alone
            assert not bool((changed & ~want).any()), j
            assert bool(changed[want][-40:].any()), j
        else:
            assert torch.equal(changed, want), (j, (changed != want).nonzero().flatten().tolist())


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("what", ["sink", "loop", "side", "cap"])
def test_small_print_matters(what, target):
    """Weights that only one mechanism reads, made large: leaving it out would show far beyond rounding."""
    name, n = "mixed", 50
    cfg, w = CONFIGS[name], dict(weights(name))
    if what == "sink":
        w["l2.mix.sink"] = torch.tensor([6.0, -9.0, 3.0]).bfloat16()
    elif what == "loop":
        w["loop.step"] = 4 * w["loop.step"]
    elif what == "side":
        w["l3.side.norm"], w["l5.side.norm"] = 4 * w["l3.side.norm"], 4 * w["l5.side.norm"]
    else:
        w["l0.mix.i.b"] = torch.tensor([40.0, -40.0, 5.0]).bfloat16()
    want = oracle.forward(cfg, w, tokens(name, n))
    # (an input gate at its cap divides by differences of large terms: bf16 projections show)
    close(engine(cfg, target, w).feed([("r", tokens(name, n), range(n))]), want, target, what, spread=3.0 if what == "cap" else 1.0)
    assert float(errors(want_logits(name, n), want).median()) > 0.1


# ---------------------------------------------------------------------------------- batches, pages, slots
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_requests_in_one_batch(name, target):
    """Portions beside decoded tokens, requests left out of steps; pages and state slots change hands, and whatever earlier
    owners left in them must not show."""
    eng = engine(name, target, num_blocks=26)
    for lc in eng.stages[0].pool.caches():
        for t in (lc.k, lc.v, lc.rec_state):
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
                                dict(stage_layers=[(0, 3), (3, 5), (5, 6)])], ids=["plain", "slices", "prefix-cache", "stages"])
def test_greedy_generation(target, kw):
    """More requests than the batch holds; with the prefix cache, requests resume from snapshots of the memories' state (of
    every pass) at a block's end."""
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


# ---------------------------------------------------------------------------------- configuration, loading, refit
def write_model(tmp_path, name):
    from safetensors.torch import save_file

    (tmp_path / "config.json").write_text(json.dumps(CONFIGS[name]))
    save_file(weights(name), str(tmp_path / "model.safetensors"))
    return str(tmp_path)


def test_loader_selects_a_stages_tensors(tmp_path):
    path = write_model(tmp_path, "mixed")
    a, b = set(ShardLoader(path, 0, 3).load_weights()), set(ShardLoader(path, 3, 6).load_weights())
    assert {"embed", "l0.mix.q", "l1.mix.left.q", "l2.mix.dq.norm"} <= a and not any(k.startswith("l3.") for k in a)
    assert {"final.norm", "final.norm.alpha", "head", "l3.mix.right.f.b", "l5.mlp.e4.down"} <= b and "embed" not in b
    assert a | b == set(weights("mixed")) and a & b == {"side.embed", "loop.step"}


def edited(path, value):
    cfg = json.loads(json.dumps(MIXED))
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return cfg


def test_config_errors():
    for path, value, text in ((("layers", 0, "type"), "something_else", "something_else"),
                              (("layers", 0, "mlp", "kind"), "other", "other"),
                              (("layers", 1, "mixer", "left", "kv_heads"), 4, "evenly"),
                              (("layers", 0, "mixer", "gate_cap"), 0.0, "gate cap"),
                              (("layers", 2, "mixer", "rot", "dims"), 10, "rotary"),
                              (("loop", "stop"), 7, "no loop"), (("loop", "times"), 0, "no loop"),
                              (("layers", 1, "mlp", "router", "top"), 7, "to choose from")):
        with pytest.raises(ValueError, match=text):
            config_from_hf(edited(path, value))
    cfg = config_from_hf(MIXED)
    assert [cfg.layer_kind(i) for i in range(6)] == ["linear", "attention", "mla_attention", "attention", "mla_attention", "linear"]
    assert [cfg.layer_passes(i) for i in range(6)] == [1, 2, 2, 1, 1, 1] and cfg.linked_layers == [(0, 2)]
    assert cfg.kv_dims(1) == (2, 64) and cfg.latent_dims(2) == (24, 8) and cfg.has_linear_layers and cfg.needs_ids_everywhere
    assert (cfg.slot_dims(2), cfg.layer_window(1), cfg.layer_window(4)) == (None, 20, 0)
    assert not config_from_hf(PLAIN).needs_ids_everywhere and config_from_hf(EQUAL).linked_layers == []
    short = {k: v for k, v in weights("mixed").items() if k != "l4.norm1b.alpha"}
    with pytest.raises(KeyError, match="l4.norm1b.alpha"):
        Engine(cfg, device="cpu", num_blocks=8, weights=short)
    wrong = dict(weights("mixed"), **{"side.embed": torch.zeros(83, 10)})
    with pytest.raises(ValueError, match="side.embed"):
        Engine(cfg, device="cpu", num_blocks=8, weights=wrong)
    for cut in ([(0, 2), (2, 6)], [(0, 1), (1, 6)]):
        with pytest.raises(ValueError, match="one pipeline stage"):
            Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), stage_layers=cut)
    with pytest.raises(ValueError, match="quantised pages"):
        Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), kv_cache_dtype="fp8_e4m3")
    from parallax_b200.models.registry import build_stage

    with pytest.raises(ValueError, match="tensor parallelism"):
        build_stage(cfg, 0, 6, "cpu", torch.float32, tp_size=2)
    with pytest.raises(ValueError, match="expert parallelism"):
        build_stage(cfg, 0, 6, "cpu", torch.float32, ep_size=2)
    with pytest.raises(ValueError, match="LoRA"):
        Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), lora={"max_loaded": 1, "paths": {}})


def test_cluster_model_info_of_a_layer_list_config():
    from parallax_b200.backend.static_config import model_info_from_config

    info = model_info_from_config(MIXED, "x")
    assert (info.num_layers, info.hidden_dim, info.vocab_size, info.num_attention_heads) == (6, 48, 83, 6)
    assert info.num_local_experts == 6 and info.num_experts_per_tok == 3


def test_sizes_of_pages_and_slots():
    """Every pass over a looped layer has pages and slots of its own, and they count."""
    from parallax_b200.cache.kv_pool import KVPool, bytes_per_block, bytes_per_linear_slot
    from parallax_b200.models.layer_spec import memory_words

    cfg = config_from_hf(MIXED)
    pool = KVPool(cfg, 0, 6, 7, 16, "cpu", torch.float32, num_linear_slots=3)
    assert [len(lc.passes) for lc in pool.layers] == [1, 2, 2, 1, 1, 1] and len(pool.caches()) == 8
    ptrs = [t.data_ptr() for lc in pool.caches() for t in (lc.k, lc.rec_state) if t is not None]
    assert len(set(ptrs)) == len(ptrs)
    per_token = 2 * (2 * 2 * 64) + 2 * 32 + 2 * 64 + 64
    assert bytes_per_block(cfg, 0, 6, 16, 4) == 16 * 4 * per_token
    assert cfg.kv_bytes_per_token_per_layer(4) == -(-4 * per_token // 6)
    words = 3 * memory_words(16, 8) + 2 * 2 * memory_words(24, 40) + 3 * memory_words(8, 16) + memory_words(32, 48)
    assert bytes_per_linear_slot(cfg, 0, 6, 4) == 4 * words
    assert 3 * bytes_per_linear_slot(cfg, 0, 6, 4) + 7 * bytes_per_block(cfg, 0, 6, 16, 4) == pool.nbytes()
    for t in pool._slot_tensors():
        t[1].fill_(5.0)
    pool.copy_slot(2, 1)
    pool.zero_slot(1)
    assert len(pool._slot_tensors()) == 5
    assert all(bool((t[2] == 5).all()) and bool((t[1] == 0).all()) for t in pool._slot_tensors())


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("stages", [None, [(0, 3), (3, 4), (4, 6)]])
def test_refit(target, stages):
    name, n = "mixed", 40
    eng = engine(name, target, stage_layers=stages)
    other = oracle.random_weights(CONFIGS[name], seed=77)
    eng.update_weights({k: v for k, v in other.items() if not k.startswith("l2.")})
    new = {k: (weights(name) if k.startswith("l2.") else other)[k] for k in other}
    close(eng.feed([("r", tokens(name, n), range(n))]), oracle.forward(CONFIGS[name], new, tokens(name, n)), target)
    eng.release_fed("r")
    eng.update_weights({k: v for k, v in weights(name).items() if k.startswith(("l3.", "l5."))})     # layers without the tables
    new = {k: (weights(name) if k.startswith(("l2.", "l3.", "l5.")) else other)[k] for k in other}
    close(eng.feed([("r", tokens(name, n), range(n))]), oracle.forward(CONFIGS[name], new, tokens(name, n)), target)


@pytest.mark.parametrize("name", ["tiny-zasalix", "small-zasalix"])
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
