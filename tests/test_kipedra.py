"""Kipedra through the engine (loader, caches, scheduler, sampling, replay tool) against ``kipedra_oracle``."""
import io
import json
import random
import sys

import numpy as np
import pytest
import torch

import kipedra_oracle as O
from decoder_harness import (be, check, expected, feed, generate, replay_for, requests, runner_for, sure_prompts,  # noqa: F401
                             tokens)
from tgi_b200.utils import synthetic as syn

A, D, dense, moe = syn.kipedra_attention, syn.kipedra_delta, syn.kipedra_dense, syn.kipedra_moe

CONFIGS = {
    # both mixers, dense and routed, layers without feed-forward, a loop in the middle that holds both kinds of cache
    "mixed": syn.kipedra_config([
        A(window=24, mlp=dense()), D(mlp=moe()), A(heads=6, kv_heads=3, dim=64, vdim=64, window=37, rot_dims=24, conv=3),
        D(heads=3, kv_heads=1, dim=32, vdim=20, mlp=dense(40)), A(window=9, base=300.0, mlp=moe(experts=6, top=2, scale=0.7))],
        loop=(1, 4, 2)),
    # the loop is the whole model, three times; sizes that are no multiple of 8, other taps
    "odd": syn.kipedra_config([
        D(heads=2, kv_heads=2, dim=36, vdim=12, conv=5, mlp=moe(ff=21, experts=5, top=1)),
        A(heads=3, kv_heads=1, dim=20, vdim=52, window=33, rot_dims=12, scale=0.4, conv=2, mlp=dense(50))],
        width=100, vocab=131, eps=1e-3, residual_mult=0.25, loop=(0, 2, 3)),
    # every expert for every token: no choice that rounding could tip; head sizes of the tensor-core kernels; no loop
    "all": syn.kipedra_config([
        A(heads=4, kv_heads=2, dim=128, vdim=128, window=64, mlp=moe(experts=4, top=4)),
        A(heads=4, kv_heads=1, dim=128, vdim=96, window=37, rot_dims=64, mlp=dense(200)),
        D(heads=4, kv_heads=2, dim=64, vdim=96, conv=3, mlp=moe(ff=24, experts=3, top=3, scale=1.0))], width=128, residual_mult=1.0),
    # no page is ever read
    "recurrent": syn.kipedra_config([D(heads=4, kv_heads=2, dim=64, vdim=32), D(heads=1, kv_heads=1, dim=16, vdim=16, mlp=dense(64))],
                                    width=64, residual_mult=0.7, loop=(1, 2, 4)),
}
# layers whose expert choice can hang on a rounding
CLOSE = {"mixed", "odd"}
SEEDS = {"mixed": 3, "odd": 1, "all": 3, "recurrent": 2}

_CKPT = {}


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    def get(name):
        if name not in _CKPT:
            cfg = CONFIGS[name]
            sd = {k: v.to(torch.bfloat16) for k, v in syn.kipedra_state_dict(cfg, seed=SEEDS[name]).items()}
            _CKPT[name] = (cfg, sd, syn.write_checkpoint(tmp_path_factory.mktemp(name), cfg, sd), {}, O)
        return _CKPT[name]

    return get


def free_again(rp):
    assert rp.pages.available == rp.pages.capacity and rp.runner.state_slots.available == 4


@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_portions_and_decoding(be, checkpoints, name):
    ck = checkpoints(name)
    ids = tokens(ck[0], 150, 1)
    want = expected(ck, ids)
    rp = replay_for(ck, be, 192)
    for portions in ([150], [1] * 150, [2] * 75, [1, 2, 46, 1, 50, 2, 2, 16, 15, 1, 14], [100] + [1] * 50, [47, 3, 60, 40]):
        check(feed(rp, "a", ids, portions), want, be[1], name in CLOSE)
        free_again(rp)


@pytest.mark.parametrize("name", ["mixed", "odd", "all"])
def test_layer_runs_one_by_one(be, checkpoints, name):
    """The residual stream after every run of a layer, so that a difference names its layer and pass."""
    from tgi_b200 import ops
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch

    ck = checkpoints(name)
    ids = tokens(ck[0], 60, 2)
    layers = []
    O.forward(ck[0], ck[1], ids, layers)
    rp = replay_for(ck, be, 64)
    r = rp.runner
    assert len(r.kv_cache) == len(r.model.layer_runs) == len(layers) > len(r.model.layers) - (name == "all")
    seq = rp._admit()
    rp._extend(seq, ids)
    meta, _ = r.build_meta(FlashCausalLMBatch(0, [seq], None, r.device), [60], [[0]])
    residual, h = ops.embed_residual(meta.input_ids, r.model.embed.weight), None
    for i, (layer, cache) in enumerate(zip(r.model.layer_runs, r.kv_cache)):
        h, residual = layer(h, residual, meta, None, cache)
        assert residual.dtype == torch.float32
        after = residual + ck[0]["residual_mult"] * sum(x.float() for x in (h if isinstance(h, tuple) else (h,)))
        err = (after.double().cpu() - layers[i]).pow(2).mean(-1).sqrt() / layers[i].std()
        if be[1] == torch.float32 or name not in CLOSE:
            assert err.max() < (2e-5 if be[1] == torch.float32 else 0.03), (i, err)
        else:       # an expert choice tipped by a rounding stays in the stream for many tokens
            assert err.quantile(0.25) < 0.03, (i, err)


@pytest.mark.parametrize("name", ["mixed", "odd", "all"])
def test_batches_of_unequal_requests(be, checkpoints, name):
    """Up to four live requests in one batch, portions beside single tokens, requests left out of steps, pages and slots
    handed on from finished requests; every logit as if the request were alone."""
    ck = checkpoints(name)
    rp = replay_for(ck, be, 4 * 80)
    rng = random.Random(5)
    waiting = [(f"r{i}", tokens(ck[0], n, 10 + i)) for i, n in enumerate((70, 1, 33, 80, 49, 2, 64, 17, 77))]
    live, seen_pages, seen_slots, gots, wants = {}, [], [], [], []
    while waiting or live:
        while waiting and len(live) < 4:
            n, ids = waiting.pop(0)
            live[n] = [ids, 0]
        entries, end, want = [], [], []
        for n, (ids, at) in list(live.items()):
            if rng.random() < 0.2 and len(live) > 1:
                continue
            k = min(len(ids) - at, rng.choice([1, 1, 1, 2, 3, 16, 31]))
            entries.append({"id": n, "tokens": ids[at:at + k], "want": list(range(k))})
            want.append(expected(ck, ids)[at:at + k])
            live[n][1] += k
            if live[n][1] == len(ids):
                end.append(n)
                del live[n]
        if not entries:
            continue
        rng.shuffle(order := list(range(len(entries))))
        gots.append(rp.step([entries[i] for i in order], []))
        wants.append(torch.cat([want[i] for i in order]))
        for n in end:
            seen_pages.append(set(rp.live[n].blocks))
            seen_slots.append(rp.live[n].state.unit)
            rp.end(n)
    check(torch.cat(gots), torch.cat(wants), be[1], name in CLOSE)
    assert len(seen_slots) > len(set(seen_slots)) and sum(map(len, seen_pages)) > len(set.union(*seen_pages))
    free_again(rp)


def test_passes_of_a_loop_have_their_own_cache(be, checkpoints):
    """Two passes over one layer: cutting the prompt or sharing one cache between the passes would change what the second
    pass finds; the caches of the passes hold different values."""
    ck = checkpoints("recurrent")
    ids = tokens(ck[0], 40, 3)
    rp = replay_for(ck, be, 64)
    check(feed(rp, "a", ids, [1, 20, 1, 18], end=False), expected(ck, ids), be[1])
    slot = rp.live["a"].state.unit
    assert [len(c) for c in rp.runner.kv_cache] == [2] * 5
    states = [c[1][slot].float().cpu() for c in rp.runner.kv_cache[1:]]
    for a, b in zip(states, states[1:]):
        assert (a - b).abs().max() > 1e-2 * a.abs().max()
    rp.end("a")


def test_first_tokens(be, checkpoints):
    """Nothing comes before a sequence: one- to five-token prompts, alone, on a slot whose last request left a past."""
    ck = checkpoints("all")
    rp = replay_for(ck, be, 64)
    feed(rp, "old", tokens(ck[0], 33, 8), [33])
    for n in range(1, 6):
        ids = tokens(ck[0], n, 20 + n)
        for portions in ([n], [1] * n):
            check(feed(rp, "a", ids, portions), expected(ck, ids), be[1])


def test_long_decoding(be, checkpoints):
    """Hundreds of single tokens, over many pages and windows."""
    ck = checkpoints("all")
    ids = tokens(ck[0], 330, 9)
    rp = replay_for(ck, be, 384)
    check(feed(rp, "a", ids, [2] + [1] * 328), expected(ck, ids), be[1])


# ---- generation ----------------------------------------------------------------------------------
_SURE = {}


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation(be, checkpoints, graphs):
    ck = checkpoints("all")
    if not _SURE:
        _SURE["all"] = sure_prompts(ck, 3, 30, 6)
    cases = _SURE["all"]
    runner = runner_for(ck, be)
    prompts, new = [c[0] for c in cases], [6, 4, 6]
    if graphs:
        if be[0].type != "cuda":
            pytest.skip("graphs exist on the GPU only")
        from tgi_b200.models.graphs import DecodeGraphs

        init = runner.init_kv_cache

        def init_and_capture(*a, **k):       # captured on the cache that `generate` makes
            init(*a, **k)
            runner.graphs = DecodeGraphs(runner, 96, buckets=[1, 2, 4])
            runner.graphs.capture_all()

        runner.init_kv_cache = init_and_capture
    want = {i: c[1][:n] for i, (c, n) in enumerate(zip(cases, new))}
    assert generate(runner, prompts, new) == want
    assert generate(runner, prompts, new, max_prefill=13) == want        # prompts in portions beside decoded tokens
    assert generate(runner, prompts, new, max_prefill=20, late=(1,)) == want
    assert runner.state_slots.available == 3


@pytest.mark.gpu
def test_warmup_then_generation(checkpoints, monkeypatch):
    """The server's start: a first step sizes pages and slots and captures the decode steps; generation on them."""
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch as B
    from tgi_b200.proto import generate_v3 as pb

    monkeypatch.setenv("CUDA_MEMORY_FRACTION", "0.1")
    monkeypatch.setenv("CUDA_GRAPHS", "1,2,4")
    ck = checkpoints("all")
    if not _SURE:
        _SURE["all"] = sure_prompts(ck, 3, 30, 6)
    r = runner_for(ck, (torch.device("cuda"), torch.bfloat16))
    reqs, _ = requests([tokens(ck[0], 60, 1)], [4])
    del reqs[0].blocks[:]
    cap, _, total = r.warmup(B.from_tokenized(pb.Batch(id=0, requests=reqs, size=1), [tokens(ck[0], 60, 1)], r.tokenizer, r.dtype,
                                              r.device), 64, 96)
    assert cap >= total == 96 and r.graphs is not None and r.state_slots.available == r.max_batch_size
    r.init_kv_cache = lambda *a, **k: None       # generate on the cache that was captured
    cases = _SURE["all"]
    assert generate(r, [c[0] for c in cases], [6] * 3, late=(2,)) == {i: c[1] for i, c in enumerate(cases)}
    assert r.state_slots.available == r.max_batch_size


def test_attention_layers_alone_still_hold_slots(tmp_path):
    """Short convolutions make a state: an attention-only model has slots, keeps no prefixes, and is not run ahead."""
    from tgi_b200.models import get_model
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch as B
    from tgi_b200.proto import generate_v3 as pb

    cfg = syn.kipedra_config([A(window=12, mlp=dense(40))], width=64, loop=(0, 1, 2))
    path = syn.write_checkpoint(tmp_path / "m", cfg, syn.kipedra_state_dict(cfg, seed=4))
    r = get_model(str(path), dtype="float32", device=torch.device("cpu"), max_positions=128)
    assert r.recurrent and not r.info.use_prefix_caching and r.info.max_batch_size == r.max_batch_size > 0 and not r.overlap_decode
    per_token = 2 * 2 * (32 + 16) * 4                # two passes, two heads, keys and values, fp32
    assert r.kv_bytes_per_block() == r.block_size * per_token
    prompts = [tokens(cfg, n, n) for n in (9, 12, 5)]
    reqs, blocks = requests(prompts, [4, 4, 4])
    r.init_kv_cache(blocks, state_slots=3)
    make = lambda: B.from_tokenized(pb.Batch(id=0, requests=reqs, size=3), prompts, r.tokenizer, r.dtype, r.device)
    _, batch, _ = r.generate_token(make())
    assert r.state_slots.available == 0
    with pytest.raises(RuntimeError, match="recurrent state slots"):
        r.generate_token(make())
    batch = batch.filter([2])
    assert r.state_slots.available == 2
    del batch
    assert r.state_slots.available == 3
    lost = make()
    lost.seqs[0].cache_len = 4
    with pytest.raises(RuntimeError, match="without its recurrent state"):
        r.generate_token(lost)


def test_sampling_and_logprobs_use_the_same_path(checkpoints):
    """Prompt log-probabilities and a sampled continuation come out of the engine as for its other models."""
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch as B
    from tgi_b200.proto import generate_v3 as pb

    ck = checkpoints("mixed")
    r = runner_for(ck, (torch.device("cpu"), torch.float32))
    ids = tokens(ck[0], 20, 4)
    reqs, blocks = requests([ids], [3])
    reqs[0].prefill_logprobs = True
    reqs[0].parameters.do_sample, reqs[0].parameters.seed, reqs[0].parameters.top_k = True, 7, 5
    r.init_kv_cache(blocks, state_slots=1)
    batch = B.from_tokenized(pb.Batch(id=0, requests=reqs, size=1), [ids], r.tokenizer, r.dtype, r.device)
    gens, batch, _ = r.generate_token(batch)
    lp = torch.log_softmax(expected(ck, ids), -1)
    assert np.allclose(gens[0].prefill_tokens.logprobs[1:], lp[torch.arange(19), torch.tensor(ids[1:])].numpy(), atol=1e-4)
    assert gens[0].tokens.token_ids[0] in expected(ck, ids)[-1].topk(5).indices.tolist()
    while batch is not None:
        gens, batch, _ = r.generate_token(batch)
    assert gens[0].generated_text is not None


# ---- configuration, tool, server -----------------------------------------------------------------
def test_config_reader():
    from tgi_b200.models.arch import ModelConfig, arch_for, derive_dims

    cfg = ModelConfig(CONFIGS["mixed"])
    assert cfg.model_type == "kipedra" and cfg.vocab_size == 203
    d = derive_dims(cfg, arch_for(cfg.model_type), 1)
    assert [s.kind for s in d.mixers] == ["attention", "delta", "attention", "delta", "attention"]
    assert d.layer_order == [0, 1, 2, 3, 1, 2, 3, 4] and d.residual_scale == 0.4 and d.eps == 1e-5
    assert [s.window for s in d.mixers] == [24, 0, 37, 0, 9] and d.mixers[4].rot_base == 300.0 and d.mixers[2].rot_dims == 24
    assert [s.ff for s in d.mixers] == [96, 0, 0, 40, 0] and [s.feed_forward for s in d.mixers] == [True, True, False, True, True]
    assert (d.mixers[4].moe.experts, d.mixers[4].moe.top, d.mixers[4].moe.scale) == (6, 2, 0.7)
    assert all(s.recurrent for s in d.mixers) and [s.paged for s in d.mixers] == [True, False, True, False, True]
    with pytest.raises(NotImplementedError):
        derive_dims(cfg, arch_for(cfg.model_type), 2)
    for where, value in ((("layers", 0, "type"), "unheard_of"), (("layers", 0, "mlp", "kind"), "unheard_of")):
        bad = json.loads(json.dumps(CONFIGS["mixed"]))
        at = bad
        for key in where[:-1]:
            at = at[key]
        at[where[-1]] = value
        with pytest.raises(NotImplementedError):
            ModelConfig(bad)
    for loop in ({"start": 2, "stop": 9, "times": 2}, {"start": 3, "stop": 1, "times": 2}, {"start": 0, "stop": 1, "times": 0}):
        with pytest.raises(ValueError):
            ModelConfig(dict(CONFIGS["mixed"], loop=loop))
    assert ModelConfig(dict(CONFIGS["mixed"], loop=None)).layer_order == list(range(5))


def test_refused_options(checkpoints):
    from tgi_b200.models import get_model

    path = str(checkpoints("recurrent")[2])
    cpu = torch.device("cpu")
    for kw in ({"quantize": "fp8"}, {"kv_cache_dtype": "fp8_e4m3fn"}, {"dtype": "float16"}):
        with pytest.raises(NotImplementedError):
            get_model(path, device=cpu, **kw)
    with pytest.raises(ValueError, match="rolled back"):
        get_model(path, device=cpu, speculate=2)


def test_replay_tool(checkpoints, tmp_path, monkeypatch, capsys):
    from tgi_b200.server import replay

    ck = checkpoints("odd")
    ids = tokens(ck[0], 12, 6)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:7], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": ids[7:11], "want": [3, 0]},
                                     {"id": "y", "tokens": ids[:2], "want": [1]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": ids[11:], "want": [0]}], "end": ["x"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(map(json.dumps, steps)) + "\n"))
    assert replay.main(["--model", str(ck[2]), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128",
                        "--device", "cpu"]) == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1", "done", "2"]
    assert not (tmp_path / "0.f32").exists()
    want = expected(ck, ids)
    got = [torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, 131)) for i in (1, 2)]
    check(got[0], torch.stack([want[10], want[7], want[1]]), torch.float32)
    check(got[1], want[11:], torch.float32)


def test_served_by_router_and_shard(tmp_path):
    """Router and shard processes: concurrent requests, more than there are state slots, prompts longer than a prefill
    step; every answer is the greedy continuation of its prompt alone."""
    import os
    import signal
    import subprocess
    import time
    from concurrent.futures import ThreadPoolExecutor

    from test_router_e2e import ROOT, _free_port, _get, _post
    from tgi_b200.router.build import build

    router_bin = build()
    cfg = syn.kipedra_config([A(window=24, mlp=dense()), D(mlp=moe()), A(window=7)], width=64, vocab=300, loop=(0, 2, 2))
    sd = syn.kipedra_state_dict(cfg, seed=3)
    path = syn.write_checkpoint(tmp_path / "m", cfg, sd)
    prompts = ["hello world", "a", "the quick brown fox jumps over the lazy dog, twice", "recurrent", "0123456789" * 4]
    n = 4
    want = [O.greedy(cfg, sd, [b + 3 for b in p.encode()], n) for p in prompts]
    uds, port = str(tmp_path / "s"), _free_port()
    env = dict(os.environ, PYTHONPATH=ROOT, TGI_B200_CPU_KV_BLOCKS="64", TGI_B200_STATE_SLOTS="2", CUDA_VISIBLE_DEVICES="",
               VIRTUAL_ENV=os.environ.get("VIRTUAL_ENV", sys.prefix))
    shard = subprocess.Popen([sys.executable, "-m", "tgi_b200.server.cli", "serve", str(path), "--uds-path", uds,
                              "--dtype", "float32"], env=env, cwd=ROOT)
    router = subprocess.Popen([str(router_bin), "--master-shard-uds-path", uds, "--tokenizer-name", str(path), "--port",
                               str(port), "--hostname", "127.0.0.1", "--max-input-tokens", "64", "--max-total-tokens", "96",
                               "--max-batch-prefill-tokens", "64", "--repo-root", ROOT], env=env, cwd=ROOT,
                              stderr=subprocess.PIPE, text=True)
    try:
        deadline = time.time() + 120
        while time.time() < deadline:
            assert shard.poll() is None and router.poll() is None
            try:
                if _get(port, "/health")[0] == 200:
                    break
            except Exception:
                time.sleep(0.3)
        ask = lambda p: _post(port, "/generate", {"inputs": p, "parameters": {"max_new_tokens": n, "details": True}})
        with ThreadPoolExecutor(5) as ex:
            answers = list(ex.map(ask, prompts))
        for (st, _, body), w in zip(answers, want):
            assert st == 200, body
            got = [t["id"] for t in json.loads(body)["details"]["tokens"]]
            assert got == w[:len(got)] and (len(got) == n or got[-1] == 2)
    finally:
        for p in (router, shard):
            p.send_signal(signal.SIGTERM)
        for p in (router, shard):
            try:
                p.wait(timeout=20)
            except subprocess.TimeoutExpired:
                p.kill()
    assert "limited to 2 requests" in router.stderr.read()
