"""Piburax through the framework's own engine against the plain restatement in ``helpers/latent_oracle.py``, on CPU
(fp32) and on a B200 (fp32 and bf16): whole prompts, decoding, portions, mixed batches, pages used again, greedy
generation through the scheduler, pipeline stages, refit, loading and the trace runner."""

import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from helpers import latent_oracle as oracle
from parallax_b200.engine.engine import Engine
from parallax_b200.engine.request import Request, SamplingParams
from parallax_b200.loader.shard_loader import ShardLoader
from parallax_b200.models.config import config_from_hf, named_config


def L(**kw):
    return dict(dict(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, scale=0.3, window=21, base=500.0, ff=72, limit=1.1), **kw)


# layers that differ in everything; windows below, at and above a page; one layer without a feed-forward
MIXED = oracle.random_config([L(), L(heads=4, dim=8, rot_dim=16, vdim=8, kv_rank=24, window=16, base=1e4, ff=None),
                              L(heads=1, dim=32, rot_dim=8, vdim=48, kv_rank=64, window=50, scale=0.11, ff=200, limit=0.7)])
# sizes that no vector or tile width divides
ODD = oracle.random_config([L(heads=3, dim=7, rot_dim=6, vdim=5, kv_rank=19, window=5, ff=33),
                            L(heads=2, dim=5, rot_dim=2, vdim=11, kv_rank=10, window=33, ff=14)],
                           vocab=37, width=30, bigram=(11, 1, 1), mult=0.5, emb_scale=1.0, eps=1e-3)
# equal sizes everywhere, no bigram table, a window of one (a token sees itself only) and one that never ends
EQUAL = oracle.random_config([L(heads=4, dim=32, rot_dim=32, vdim=32, kv_rank=32, window=1, ff=64),
                              L(heads=4, dim=32, rot_dim=32, vdim=32, kv_rank=32, window=1000, ff=64)],
                             vocab=64, width=64, bigram=None)
# tensor-core widths: several latent chunks, more heads than a query tile holds
WIDE = oracle.random_config([L(heads=8, dim=64, rot_dim=64, vdim=64, kv_rank=512, window=70, ff=256, scale=0.08),
                             L(heads=136, dim=8, rot_dim=8, vdim=8, kv_rank=136, window=40, ff=128, scale=0.2)],
                            vocab=200, width=128)
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


def close(got, want, target, what=""):
    got, want = got.double().cpu(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    err = float((d.pow(2).mean(-1).sqrt() / want.std(-1)).max())
    assert err < (2e-5 if target[1] == torch.float32 else 4e-2), (what, err)


# ---------------------------------------------------------------------------------- whole prompts and layers
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(name, target):
    eng = engine(name, target)
    for n in (1, 2, 16, 17, 113):
        got = eng.feed([("r", tokens(name, n), range(n))])
        close(got, want_logits(name, 113)[:n], target, n)
        eng.release_fed("r")
    assert eng.cache.num_free_blocks() == 40


@pytest.mark.parametrize("target", TARGETS)
def test_residual_after_every_layer(target):
    name, n = "mixed", 60
    ref = []
    oracle.forward(CONFIGS[name], weights(name), tokens(name, n), ref)
    eng = engine(name, target, stage_layers=[(0, 1), (1, 2), (2, 3)])
    seen = []
    eng.wire_hook = lambda h: (seen.append(h.clone()), h)[1]      # hidden states between pipeline stages
    close(eng.feed([("r", tokens(name, n), range(n))]), want_logits(name, n), target)
    assert len(seen) == 2 and all(h.dtype == torch.float32 for h in seen)
    for h, x in zip(seen, ref):
        tol = 2e-5 if target[1] == torch.float32 else 3e-2
        assert float((h.double().cpu() - x).norm() / x.norm()) < tol


# ---------------------------------------------------------------------------------- decoding and portions
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_decoding_equals_the_prompt(name, target):
    """Token by token from the first token on: over page borders, past every window."""
    n = 118
    eng, seq = engine(name, target), tokens(name, n)
    got = torch.cat([eng.feed([("r", [t], [0])]) for t in seq])
    close(got, want_logits(name, n), target)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("cut", [(2,), (3, 1, 5), (16,), (15, 17, 1, 1, 31), (64, 2)])
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
    """Many times the windows' length, from a short prompt."""
    name, n = "mixed", 330
    eng, seq = engine(name, target), tokens(name, n)
    eng.feed([("r", seq[:3], [])])
    got = torch.cat([eng.feed([("r", [t], [0])]) for t in seq[3:]])
    close(got, want_logits(name, n)[3:], target)


# ---------------------------------------------------------------------------------- batches, pages, slots
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_requests_in_one_batch(name, target):
    """Portions beside decoded tokens, requests left out of steps; pages and slots change hands, and whatever earlier
    owners left in them must not show."""
    eng = engine(name, target, num_blocks=26)
    for lc in eng.stages[0].pool.layers:
        lc.k.fill_(37.0)                      # what a page held before it was handed out
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


def test_feed_refuses_what_it_cannot_run():
    eng = engine("mixed", ("cpu", torch.float32), num_blocks=2)
    with pytest.raises(ValueError):
        eng.feed([("r", [1, 2], [2])])
    with pytest.raises(ValueError):
        eng.feed([("r", [10 ** 6], [])])
    with pytest.raises(ValueError):
        eng.feed([("r", tokens("mixed", 400) + [1], [])])       # longer than the engine's requests may be
    with pytest.raises(RuntimeError):
        eng.feed([("r", tokens("mixed", 40), [])])              # more pages than there are
    with pytest.raises(ValueError):
        eng.release_fed("r")
    assert eng.cache.num_free_blocks() == 2


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
@pytest.mark.parametrize("kw", [dict(), dict(chunked_prefill_size=7), dict(enable_prefix_cache=True, chunked_prefill_size=20),
                                dict(stage_layers=[(0, 2), (2, 3)])], ids=["plain", "slices", "prefix-cache", "stages"])
def test_greedy_generation(target, kw):
    """More requests than the batch holds; shared prefixes when the prefix cache is on (the first computed token then
    follows a cached one)."""
    name, n_new = "mixed", 9
    kw = dict(dict(max_requests=None, max_num_tokens_per_batch=60), **kw)
    eng = engine(name, target, **kw)
    base = tokens(name, 70, 9)
    prompts = [base[:33], tokens(name, 1, 5), base[:48], tokens(name, 27, 6), base[:64], base[:32] + tokens(name, 3, 7)]
    outs, _ = generate(eng, prompts, n_new)
    again, cached = generate(eng, prompts, n_new)
    assert (cached >= 32 * 4) == bool(kw.get("enable_prefix_cache"))
    for p, got, got2 in zip(prompts, outs, again):
        want, margins = oracle.greedy(CONFIGS[name], weights(name), p, n_new)
        for i in range(n_new):
            if target[1] == torch.bfloat16 and margins[i] < 0.15:      # a near tie may fall either way in bf16
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
    first, last = ShardLoader(path, 0, 1), ShardLoader(path, 1, 3)
    a, b = set(first.load_weights()), set(last.load_weights())
    assert {"embed", "bigram", "l0.mix.q", "l0.norm2"} <= a and not any(k.startswith(("l1.", "l2.")) for k in a)
    assert {"final.norm", "head", "l1.mix.dkv.norm", "l2.mlp.down"} <= b and "embed" not in b
    assert a | b == set(weights("mixed")) and not a & b


def test_config_errors():
    bad = json.loads(json.dumps(MIXED))
    bad["layers"][0]["type"] = "something_else"
    with pytest.raises(ValueError, match="something_else"):
        config_from_hf(bad)
    cfg = config_from_hf(MIXED)
    assert [cfg.layer_window(i) for i in range(3)] == [21, 16, 50]
    assert [cfg.latent_dims(i) for i in range(3)] == [(40, 8), (24, 16), (64, 8)]
    short = {k: v for k, v in weights("mixed").items() if k != "l1.mix.sink"}
    with pytest.raises(KeyError, match="l1.mix.sink"):
        Engine(cfg, device="cpu", num_blocks=8, weights=short)
    wrong = dict(weights("mixed"), **{"l0.mix.uk": torch.zeros(4, 4)})
    with pytest.raises(ValueError, match="l0.mix.uk"):
        Engine(cfg, device="cpu", num_blocks=8, weights=wrong)
    from parallax_b200.models.registry import build_stage

    with pytest.raises(ValueError, match="tensor parallelism"):
        build_stage(cfg, 0, 3, "cpu", torch.float32, tp_size=2)
    with pytest.raises(ValueError, match="LoRA"):
        Engine(cfg, device="cpu", num_blocks=8, weights=weights("mixed"), lora={"max_loaded": 1, "paths": {}})


def test_cluster_model_info_of_a_layer_list_config():
    from parallax_b200.backend.static_config import model_info_from_config

    info = model_info_from_config(MIXED, "x")
    assert (info.num_layers, info.hidden_dim, info.vocab_size, info.num_attention_heads) == (3, 48, 83, 4)


@pytest.mark.parametrize("target", TARGETS)
def test_refit(target):
    name, n = "mixed", 40
    eng = engine(name, target)
    other = oracle.random_weights(CONFIGS[name], seed=77)
    eng.update_weights({k: v for k, v in other.items() if not k.startswith("l1.")})
    new = {k: (weights(name) if k.startswith("l1.") else other)[k] for k in other}
    close(eng.feed([("r", tokens(name, n), range(n))]), oracle.forward(CONFIGS[name], new, tokens(name, n)), target)


@pytest.mark.parametrize("name", ["tiny-piburax", "small-piburax"])
def test_named_configs_build(name):
    eng = Engine(named_config(name), device="cpu", num_blocks=16, max_batch_size=2)
    assert len(eng.generate([[1, 2, 3]], SamplingParams(max_new_tokens=3, temperature=0.0))[0]) == 3


def test_offline_generation_command(tmp_path):
    from parallax_b200.generate import run

    res = run(write_model(tmp_path, "mixed"), "hello", max_tokens=4, device="cpu", out=lambda _line: None)
    assert res["generated_tokens"] == 4


# ---------------------------------------------------------------------------------- trace runner
def run_trace(model, out, dtype, steps, max_tokens):
    runner = Path(__file__).resolve().parent.parent / "bin" / "trace_run"
    text = "".join(json.dumps(s) + "\n" for s in steps)
    return subprocess.run([sys.executable, str(runner), "--model", model, "--dtype", dtype, "--out", str(out), "--max-tokens",
                           str(max_tokens)], input=text, capture_output=True, text=True, timeout=300,
                          env=dict(os.environ, OMP_NUM_THREADS="2"))


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
    res = run_trace(write_model(model, name), out, dtype, steps, 128)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 4", "done 5"]
    ref, V = want_logits(name, 90), CONFIGS[name]["vocab"]
    target = ("cpu", torch.float32 if dtype == "float32" else torch.bfloat16)
    for step, places in ((0, [0, 29, 1]), (4, [30, 63, 5]), (5, [89])):
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(places), V))
        close(got, ref[places], target, step)
    assert not (out / "1.f32").exists()


def test_trace_runner_refuses_families_without_32_bit(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(named_config("tiny").raw))
    assert run_trace(str(tmp_path), tmp_path, "float32", [], 64).returncode == 3
