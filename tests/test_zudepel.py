"""Zudepel through the framework's own engine against the plain restatement in ``helpers/zudepel_oracle.py``, on CPU
(fp32) and on a B200 (fp32 and bf16): whole prompts, decoding, portions, mixed batches, pages and state slots used again,
greedy generation through the scheduler, pipeline stages, refit, loading and the trace runner."""

import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from helpers import zudepel_oracle as oracle
from helpers.zudepel_oracle import attention, dense, lightning, moe
from parallax_b200.engine.engine import Engine
from parallax_b200.engine.request import Request, SamplingParams
from parallax_b200.loader.shard_loader import ShardLoader
from parallax_b200.models.config import config_from_hf, named_config

# layers that differ in everything: own and shared keys, every feed-forward behind every mixer, or none
MIXED = oracle.random_config([
    lightning(3, 16, 8, [0.6, 0.95, 0.999], dense(72)),
    attention(6, 2, 24, 16, conv=4, rot=16, scale=0.3, mlp=moe()),
    attention(4, 2, 24, 16, conv=3, rot=24, scale=0.2, kv_from=1, mlp=dense(40)),
    lightning(2, 32, 24, [0.5, 0.98], moe(experts=5, identity=0, top=3, groups=None, shared=None)),
    attention(2, 1, 40, 56, conv=2, rot=8, base=50.0, scale=0.15, mlp=None)])
# sizes that no vector or tile width divides; shared keys read across a layer
ODD = oracle.random_config([
    attention(3, 3, 7, 5, conv=3, rot=6, scale=0.5, mlp=moe(ff=11, experts=5, identity=1, top=3, groups=(3, 2), shared=13)),
    lightning(3, 9, 7, [0.8, 0.9, 1.0], dense(33)),
    attention(6, 3, 7, 5, conv=5, rot=2, scale=0.4, kv_from=0, mlp=dense(21)),
    lightning(1, 5, 3, [0.97], None)], vocab=37, width=30, eps=1e-3)
# equal sizes everywhere, a one-tap convolution, one expert per token, no identity experts
EQUAL = oracle.random_config([
    attention(4, 4, 32, 32, conv=1, rot=32, scale=0.2, mlp=moe(ff=64, experts=4, identity=0, top=1, groups=None, shared=64)),
    lightning(4, 32, 32, [0.9] * 4, dense(64))], vocab=64, width=64)
# tensor-core widths: several chunks of the head, more query heads per key head than the decode tile holds
WIDE = oracle.random_config([
    attention(8, 2, 128, 64, conv=4, rot=64, scale=0.09, mlp=moe(ff=96, experts=10, identity=2, top=4, groups=(4, 3), shared=128)),
    lightning(2, 128, 128, [0.9, 0.995], dense(256)),
    attention(34, 2, 16, 24, conv=4, rot=16, scale=0.3, mlp=moe(ff=64, experts=30, identity=3, top=6, groups=(11, 4))),
    lightning(3, 96, 40, [0.7, 0.99, 0.999], None)], vocab=200, width=128)
CONFIGS = {"mixed": MIXED, "odd": ODD, "equal": EQUAL, "wide": WIDE}
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


def engine(name, target, **kw):
    dev, dt = target
    args = dict(page_size=16, num_blocks=40, max_batch_size=4, max_num_tokens_per_batch=512, max_total_length=400,
                enable_prefix_cache=False, max_requests=4)
    args.update(kw)
    return Engine(config_from_hf(CONFIGS[name]), device=dev, dtype=dt, weights=weights(name), **args)


def errors(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std(-1)


def close(got, want, target, what=""):
    """In bf16 a close call of a router may fall the other way: a few positions may be off, the bulk may not."""
    err = errors(got, want)
    if target[1] == torch.float32:
        assert float(err.max()) < 3e-5, (what, float(err.max()))
    else:
        assert float(err.median()) < 3e-2 and float(err.quantile(0.8)) < 8e-2 and float(err.max()) < 1.0, \
            (what, [float(err.quantile(q)) for q in (0.5, 0.8, 1.0)])


# ---------------------------------------------------------------------------------- whole prompts and layers
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(name, target):
    eng = engine(name, target)
    for n in (1, 2, 16, 17, 64, 65, 113):
        got = eng.feed([("r", tokens(name, n), range(n))])
        close(got, want_logits(name, 113)[:n], target, n)
        eng.release_fed("r")
    assert eng.cache.num_free_blocks() == 40


@pytest.mark.parametrize("target", TARGETS)
def test_residual_after_every_stage(target):
    name, n = "mixed", 60
    ref = []
    oracle.forward(CONFIGS[name], weights(name), tokens(name, n), ref)
    eng = engine(name, target, stage_layers=[(0, 1), (1, 3), (3, 4), (4, 5)])
    seen = []
    eng.wire_hook = lambda h: (seen.append(h.clone()), h)[1]      # hidden states between pipeline stages
    close(eng.feed([("r", tokens(name, n), range(n))]), want_logits(name, n), target)
    assert len(seen) == 3 and all(h.dtype == torch.float32 for h in seen)
    for h, x in zip(seen, (ref[0], ref[2], ref[3])):
        err = (h.double().cpu() - x).norm(dim=-1) / x.norm(dim=-1)
        assert float(err.quantile(0.8)) < (2e-5 if target[1] == torch.float32 else 3e-2)


# ---------------------------------------------------------------------------------- decoding and portions
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_decoding_equals_the_prompt(name, target):
    """Token by token from the first token on: over page borders, with the convolutions' first taps."""
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


# ---------------------------------------------------------------------------------- batches, pages, slots
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_requests_in_one_batch(name, target):
    """Portions beside decoded tokens, requests left out of steps; pages and state slots change hands, and whatever earlier
    owners left in them must not show."""
    eng = engine(name, target, num_blocks=26)
    for lc in eng.stages[0].pool.layers:
        for t in (lc.k, lc.v, lc.conv_state, lc.rec_state):
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
                                dict(stage_layers=[(0, 1), (1, 4), (4, 5)])], ids=["plain", "slices", "prefix-cache", "stages"])
def test_greedy_generation(target, kw):
    """More requests than the batch holds; with the prefix cache, requests resume from snapshots of the convolutions' and
    the recurrent layers' state at a block's end."""
    name, n_new = "mixed", 9
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


@pytest.mark.parametrize("target", TARGETS[:2])
def test_routed_experts_record(target):
    """Layers may choose different numbers of experts; identity experts are recorded by their router output."""
    name, n = "mixed", 30
    eng = engine(name, target, return_routed_experts=True)
    req = Request(input_ids=tokens(name, n), sampling_params=SamplingParams(max_new_tokens=2, temperature=0.0, ignore_eos=True))
    eng.add_request(req)
    while eng.has_work():
        eng.step()
    rec = torch.tensor(req.routed_experts)
    assert rec.shape == (n + 1, 2, 3)
    states, w, cfg = [], weights(name), CONFIGS[name]
    oracle.forward(cfg, w, tokens(name, n), states)
    for j, li in enumerate((1, 3)):
        want, p = [], f"l{li}."
        oracle.routed(cfg["layers"][li]["mlp"], w, p + "mlp.", oracle.rms_norm(states[li - 1], w[p + "norm1"], 1e-6), want)
        k = len(want[0])
        assert rec[:n, j, :k].tolist() == want and bool((rec[:, j, k:] == -1).all())


# ---------------------------------------------------------------------------------- configuration, loading, refit
def write_model(tmp_path, name):
    from safetensors.torch import save_file

    (tmp_path / "config.json").write_text(json.dumps(CONFIGS[name]))
    save_file(weights(name), str(tmp_path / "model.safetensors"))
    return str(tmp_path)


def test_loader_selects_a_stages_tensors(tmp_path):
    path = write_model(tmp_path, "mixed")
    first, last = ShardLoader(path, 0, 1), ShardLoader(path, 1, 5)
    a, b = set(first.load_weights()), set(last.load_weights())
    assert {"embed", "l0.mix.q", "l0.mix.norm"} <= a and not any(k.startswith("l1.") for k in a)
    assert {"final.norm", "head", "l1.mix.q.conv", "l3.mlp.e4.down"} <= b and "embed" not in b
    assert a | b == set(weights("mixed")) and not a & b


def edited(path, value):
    cfg = json.loads(json.dumps(MIXED))
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return cfg


def test_config_errors():
    for path, value, text in ((("layers", 0, "type"), "something_else", "something_else"),
                              (("layers", 2, "mixer", "kv_from"), 0, "no earlier layer"),
                              (("layers", 1, "mixer", "kv_from"), 2, "no earlier layer"),
                              (("layers", 2, "mixer", "vdim"), 24, "differ in their key"),
                              (("layers", 1, "mixer", "kv_heads"), 4, "evenly"),
                              (("layers", 0, "mixer", "decay"), [0.5], "decays"),
                              (("layers", 1, "mlp", "router", "groups", "count"), 3, "groups"),
                              (("layers", 1, "mlp", "router", "top"), 5, "to choose from")):
        with pytest.raises(ValueError, match=text):
            config_from_hf(edited(path, value))
    cfg = config_from_hf(MIXED)
    assert [cfg.layer_kind(i) for i in range(5)] == ["linear", "attention", "attention", "linear", "attention"]
    assert cfg.kv_dims(1) == (2, 64) and cfg.kv_dims(2) is None and cfg.slot_dims(2) == ((2, 4 * 24), None)
    assert cfg.slot_dims(0) == (None, (3, 16, 8)) and cfg.has_linear_layers and cfg.linked_layers == [(1, 2)]
    short = {k: v for k, v in weights("mixed").items() if k != "l1.mix.sink"}
    with pytest.raises(KeyError, match="l1.mix.sink"):
        Engine(cfg, device="cpu", num_blocks=8, weights=short)
    wrong = dict(weights("mixed"), **{"l1.mix.v.conv": torch.zeros(4, 4)})
    with pytest.raises(ValueError, match="l1.mix.v.conv"):
        Engine(cfg, device="cpu", num_blocks=8, weights=wrong)
    with pytest.raises(ValueError, match="one pipeline stage"):
        Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), stage_layers=[(0, 2), (2, 5)])
    with pytest.raises(ValueError, match="quantised pages"):
        Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), kv_cache_dtype="fp8_e4m3")
    from parallax_b200.models.registry import build_stage

    with pytest.raises(ValueError, match="tensor parallelism"):
        build_stage(cfg, 0, 3, "cpu", torch.float32, tp_size=2)
    with pytest.raises(ValueError, match="expert parallelism"):
        build_stage(cfg, 0, 3, "cpu", torch.float32, ep_size=2)
    with pytest.raises(ValueError, match="LoRA"):
        Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), lora={"max_loaded": 1, "paths": {}})


def test_cluster_model_info_of_a_layer_list_config():
    from parallax_b200.backend.static_config import model_info_from_config

    info = model_info_from_config(MIXED, "x")
    assert (info.num_layers, info.hidden_dim, info.vocab_size, info.num_attention_heads) == (5, 48, 83, 6)
    assert info.num_local_experts == 6 and info.num_experts_per_tok == 3


def test_sizes_of_pages_and_slots():
    from parallax_b200.cache.kv_pool import KVPool, bytes_per_block, bytes_per_linear_slot

    cfg = config_from_hf(MIXED)
    pool = KVPool(cfg, 0, 5, 7, 16, "cpu", torch.float32, num_linear_slots=3)
    paged = sum(t.numel() for lc in pool.layers for t in (lc.k, lc.v) if t is not None)
    assert 7 * bytes_per_block(cfg, 0, 5, 16, 4) == 4 * paged == 7 * 16 * 4 * 2 * (2 * 64 + 1 * 64)
    assert 3 * bytes_per_linear_slot(cfg, 0, 5, 4) + 7 * bytes_per_block(cfg, 0, 5, 16, 4) == pool.nbytes()
    for t in pool._slot_tensors():
        t[1].fill_(5.0)
    pool.copy_slot(2, 1)
    pool.zero_slot(1)
    assert all(bool((t[2] == 5).all()) and bool((t[1] == 0).all()) for t in pool._slot_tensors())


@pytest.mark.parametrize("target", TARGETS)
def test_refit(target):
    name, n = "mixed", 40
    eng = engine(name, target)
    other = oracle.random_weights(CONFIGS[name], seed=77)
    eng.update_weights({k: v for k, v in other.items() if not k.startswith("l2.")})
    new = {k: (weights(name) if k.startswith("l2.") else other)[k] for k in other}
    close(eng.feed([("r", tokens(name, n), range(n))]), oracle.forward(CONFIGS[name], new, tokens(name, n)), target)


@pytest.mark.parametrize("name", ["tiny-zudepel", "small-zudepel"])
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
