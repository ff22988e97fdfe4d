"""Gisilix through the engine (loader, caches, scheduler, sampling, replay tool) against ``gisilix_oracle``."""
import io
import json
import random
import sys

import numpy as np
import pytest
import torch

import gisilix_oracle as O
from decoder_harness import (be, check, expected, feed, generate, replay_for, requests, runner_for, sure_prompts,  # noqa: F401
                             tokens)
from tgi_b200.utils import synthetic as syn

A, N, R, moe = syn.gisilix_attention, syn.gisilix_latent, syn.gisilix_rotated_latent, syn.gisilix_moe
dense = syn.kipedra_dense

CONFIGS = {
    # every mixer, every feed-forward, two layers that read the keys of the first, with other gates, sinks and temperatures
    "mixed": syn.gisilix_config([
        A(mlp=dense()), R(mlp=moe()), N(mlp=dense(40)), A(heads=6, coef=0.5, every=9, softcap=3.0, kv_from=0, mlp=moe(experts=6, top=2, shared=0)),
        R(heads=6, window=37, rot_dim=12, scaling=None), A(kv_from=0)]),
    # sizes that are no multiple of 8; a source in the middle
    "odd": syn.gisilix_config([
        N(heads=3, dim=10, vdim=14, rank=30, mlp=moe(ff=21, experts=5, top=1, shared=13)),
        A(heads=3, kv_heads=1, dim=22, vdim=30, every=1, mlp=dense(50)),
        A(heads=2, kv_heads=1, dim=22, vdim=30, kv_from=1, mlp=None)], width=100, vocab=131, eps=1e-3),
    # every expert for every token: no choice that rounding could tip; head sizes of the tensor-core kernels
    "all": syn.gisilix_config([
        R(heads=8, dim=128, vdim=128, rank=512, rot_dim=64, window=70, base=5000.0, scaling=(3.0, 16.0, 1.0, 100), mlp=moe(experts=4, top=4)),
        A(heads=4, kv_heads=2, dim=128, vdim=128, every=33, softcap=12.0, mlp=dense(200)),
        N(heads=4, dim=64, vdim=96, rank=192, mlp=moe(ff=24, experts=3, top=3, shared=64)),
        A(heads=8, kv_heads=2, dim=128, vdim=128, kv_from=1, mlp=dense(72))], width=128),
}
# layers whose expert choice can hang on a rounding
CLOSE = {"mixed", "odd"}
SEEDS = {"mixed": 3, "odd": 1, "all": 3}

_CKPT = {}


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    def get(name):
        if name not in _CKPT:
            cfg = CONFIGS[name]
            sd = {k: v.to(torch.bfloat16) for k, v in syn.gisilix_state_dict(cfg, seed=SEEDS[name]).items()}
            _CKPT[name] = (cfg, sd, syn.write_checkpoint(tmp_path_factory.mktemp(name), cfg, sd), {}, O)
        return _CKPT[name]

    return get


@pytest.fixture(params=[None, 2], ids=["", "written-out"])
def expand(request, be, monkeypatch):
    """Also with keys and values written out for every portion of two tokens and more."""
    from tgi_b200.models import mixers

    if request.param is not None:
        if be[0].type != "cuda" or be[1] != torch.bfloat16:
            pytest.skip("written-out keys are a bf16 kernel")
        monkeypatch.setattr(mixers, "EXPAND_TOKENS", request.param)


def free_again(rp):
    assert rp.pages.available == rp.pages.capacity and rp.runner.state_slots is None


@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_portions_and_decoding(be, checkpoints, expand, name):
    ck = checkpoints(name)
    ids = tokens(ck[0], 150, 1)
    want = expected(ck, ids)
    rp = replay_for(ck, be, 192)
    for portions in ([150], [1] * 150, [2] * 75, [1, 2, 46, 1, 50, 2, 2, 16, 15, 1, 14], [100] + [1] * 50, [47, 3, 60, 40]):
        check(feed(rp, "a", ids, portions), want, be[1], name in CLOSE)
        free_again(rp)


@pytest.mark.parametrize("name", CONFIGS)
def test_layers_one_by_one(be, checkpoints, name):
    """The residual stream after every layer, so that a difference names its layer."""
    from tgi_b200 import ops
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch

    ck = checkpoints(name)
    ids = tokens(ck[0], 70, 2)
    layers = []
    O.forward(ck[0], ck[1], ids, layers)
    rp = replay_for(ck, be, 96)
    r = rp.runner
    seq = rp._admit()
    rp._extend(seq, ids)
    meta, _ = r.build_meta(FlashCausalLMBatch(0, [seq], None, r.device), [70], [[0]])
    residual, h = ops.embed_residual(meta.input_ids, r.model.embed.weight), None
    for i, (layer, cache) in enumerate(zip(r.model.layer_runs, r.kv_cache)):
        h, residual = layer(h, residual, meta, None, cache)
        assert residual.dtype == torch.float32
        after = residual + sum(x.float() for x in (h if isinstance(h, tuple) else (h,)))
        err = (after.double().cpu() - layers[i]).pow(2).mean(-1).sqrt() / layers[i].std()
        if be[1] == torch.float32 or name not in CLOSE:
            assert err.max() < (2e-5 if be[1] == torch.float32 else 0.03), (i, err)
        else:       # an expert choice tipped by a rounding stays in the stream for many tokens
            assert err.quantile(0.25) < 0.03, (i, err)


@pytest.mark.parametrize("name", CONFIGS)
def test_batches_of_unequal_requests(be, checkpoints, expand, name):
    """Up to four live requests in one batch, portions beside single tokens, requests left out of steps, pages handed on
    from finished requests; every logit as if the request were alone."""
    ck = checkpoints(name)
    rp = replay_for(ck, be, 4 * 96)
    rng = random.Random(5)
    waiting = [(f"r{i}", tokens(ck[0], n, 10 + i)) for i, n in enumerate((70, 1, 33, 80, 49, 2, 64, 17, 95))]
    live, seen_pages, gots, wants = {}, [], [], []
    while waiting or live:
        while waiting and len(live) < 4:
            n, ids = waiting.pop(0)
            live[n] = [ids, 0]
        entries, end, want = [], [], []
        for n, (ids, at) in list(live.items()):
            if rng.random() < 0.2 and len(live) > 1:
                continue
            k = min(len(ids) - at, rng.choice([1, 1, 1, 2, 3, 16, 31, 80]))
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
            rp.end(n)
    check(torch.cat(gots), torch.cat(wants), be[1], name in CLOSE)
    assert sum(map(len, seen_pages)) > len(set.union(*seen_pages))
    free_again(rp)


def test_shared_keys_are_held_once(be, checkpoints):
    """A layer that reads another's keys has no cache of its own and no key tensors; only latents are kept elsewhere."""
    from tgi_b200 import ops

    ck = checkpoints("mixed")
    rp = replay_for(ck, be, 64)
    r = rp.runner
    caches = r.kv_cache
    assert caches[3][0] is caches[0][0] and caches[5][1] is caches[0][1] and [len(c) for c in caches] == [2, 1, 1, 2, 1, 2]
    size = torch.empty((), dtype=be[1]).element_size()
    k, v = ops.attention_pitch(24, 16, be[1], be[0])
    widths = [ops.latent_layout(40, rot, be[1], be[0])[1] for rot in (8, 0, 12)]
    assert r.kv_bytes_per_block() == 16 * size * (2 * (k + v) + sum(widths))
    if be[0].type == "cpu":
        assert widths == [48, 40, 52]
    ids = tokens(ck[0], 40, 3)
    want = expected(ck, ids)
    changed = dict(ck[1])
    changed["l0.mix.k"] = -changed["l0.mix.k"]               # reaches the last layer's attention too
    assert (O.forward(ck[0], changed, ids) - want).abs().max() > 0.05
    check(feed(rp, "a", ids, [1, 20, 1, 18]), want, be[1], True)


def test_first_tokens(be, checkpoints):
    """Nothing comes before a sequence: one- to five-token prompts, alone, on pages whose last request left other keys."""
    ck = checkpoints("all")
    rp = replay_for(ck, be, 64)
    feed(rp, "old", tokens(ck[0], 33, 8), [33])
    for n in range(1, 6):
        ids = tokens(ck[0], n, 20 + n)
        for portions in ([n], [1] * n):
            check(feed(rp, "a", ids, portions), expected(ck, ids), be[1])


def test_long_decoding(be, checkpoints):
    """Hundreds of single tokens, over many pages, tiles, windows and steps of the temperature."""
    ck = checkpoints("all")
    ids = tokens(ck[0], 330, 9)
    rp = replay_for(ck, be, 384)
    check(feed(rp, "a", ids, [2] + [1] * 328), expected(ck, ids), be[1])


def test_prefix_of_another_request(be, checkpoints, expand):
    """Everything a layer keeps is in pages: a request starts behind a prefix that an earlier one brought."""
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch as B
    from tgi_b200.proto import generate_v3 as pb

    ck = checkpoints("all")
    r = runner_for(ck, be)
    assert r.info.use_prefix_caching and not r.recurrent and r.max_batch_size is None
    first, tail = tokens(ck[0], 64, 1), tokens(ck[0], 41, 2)
    r.init_kv_cache(16)
    for ids, cached, blocks in ((first, 0, [5, 3, 9, 1, 2]), (first[:48] + tail, 48, [5, 3, 9, 7, 8, 4, 6])):
        reqs, _ = requests([ids], [1])
        del reqs[0].blocks[:]
        reqs[0].blocks.extend(blocks)
        reqs[0].cache_len = cached
        batch = B.from_tokenized(pb.Batch(id=0, requests=reqs, size=1), [ids], r.tokenizer, r.dtype, r.device)
        counts = batch.plan_step()
        assert counts == [len(ids) - cached]
        got = r.step_logits(batch, counts, [list(range(counts[0]))]).float().cpu()
        check(got, expected(ck, ids)[cached:], be[1])


# ---- generation ----------------------------------------------------------------------------------
_SURE = {}


def sure(ck):
    if not _SURE:
        _SURE["all"] = sure_prompts(ck, 3, 30, 6)
    return _SURE["all"]


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation(be, checkpoints, graphs):
    ck = checkpoints("all")
    cases = sure(ck)
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
    assert not graphs or runner.overlap_hits > 0


@pytest.mark.gpu
def test_warmup_then_generation(checkpoints, monkeypatch):
    """The server's start: a first step sizes pages and captures the decode steps; generation on them."""
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch as B
    from tgi_b200.proto import generate_v3 as pb

    monkeypatch.setenv("CUDA_MEMORY_FRACTION", "0.1")
    monkeypatch.setenv("CUDA_GRAPHS", "1,2,4")
    ck = checkpoints("all")
    r = runner_for(ck, (torch.device("cuda"), torch.bfloat16))
    reqs, _ = requests([tokens(ck[0], 60, 1)], [4])
    del reqs[0].blocks[:]
    cap, _, total = r.warmup(B.from_tokenized(pb.Batch(id=0, requests=reqs, size=1), [tokens(ck[0], 60, 1)], r.tokenizer, r.dtype,
                                              r.device), 64, 96)
    assert cap >= total == 96 and r.graphs is not None
    r.init_kv_cache = lambda *a, **k: None       # generate on the cache that was captured
    cases = sure(ck)
    assert generate(r, [c[0] for c in cases], [6] * 3, late=(2,)) == {i: c[1] for i, c in enumerate(cases)}


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
    r.init_kv_cache(blocks)
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
    assert cfg.model_type == "gisilix" and cfg.vocab_size == 203
    d = derive_dims(cfg, arch_for(cfg.model_type), 1)
    s = d.mixers
    assert [m.kind for m in s] == ["attention", "latent", "latent", "attention", "latent", "attention"]
    assert not any(m.recurrent for m in s) and all(m.paged for m in s) and d.eps == 1e-5 and d.residual_scale == 1.0
    assert [m.kv_from for m in s] == [None, None, None, 0, None, 0] and [m.window for m in s] == [0, 24, 0, 0, 37, 0]
    assert (s[3].q_temp, s[3].softcap, s[3].out_gate) == ((0.5, 9), 3.0, "element") and s[1].out_gate == "head" and s[2].out_gate == ""
    assert s[1].rot_yarn == (4.0, 8.0, 1.0, 128.0) and s[4].rot_yarn is None and [m.rot_dims for m in s] == [0, 8, 0, 0, 12, 0]
    assert (s[1].moe.experts, s[1].moe.top, s[1].moe.ff, s[1].moe.shared_ff, s[1].moe.gated, s[1].moe.router) == (10, 3, 24, 40, True, "softmax")
    assert s[3].moe.shared_ff == 0 and [m.feed_forward for m in s] == [True, True, True, True, False, False]
    with pytest.raises(NotImplementedError):
        derive_dims(cfg, arch_for(cfg.model_type), 2)
    for where, value, error in ((("layers", 0, "type"), "unheard_of", NotImplementedError), (("layers", 0, "mlp", "kind"), "unheard_of", NotImplementedError),
                                (("layers", 3, "mixer", "kv_from"), 1, ValueError), (("layers", 3, "mixer", "kv_from"), 5, ValueError),
                                (("layers", 5, "mixer", "kv_from"), 3, ValueError), (("layers", 3, "mixer", "dim"), 32, ValueError)):
        bad = json.loads(json.dumps(CONFIGS["mixed"]))
        at = bad
        for key in where[:-1]:
            at = at[key]
        at[where[-1]] = value
        with pytest.raises(error):
            ModelConfig(bad)


def test_refused_options(checkpoints):
    from tgi_b200.models import get_model

    path = str(checkpoints("odd")[2])
    for kw in ({"quantize": "fp8"}, {"kv_cache_dtype": "fp8_e4m3fn"}, {"dtype": "float16"}):
        with pytest.raises(NotImplementedError):
            get_model(path, device=torch.device("cpu"), **kw)


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
    want = expected(ck, ids)
    got = [torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, 131)) for i in (1, 2)]
    check(got[0], torch.stack([want[10], want[7], want[1]]), torch.float32)
    check(got[1], want[11:], torch.float32)


def test_served_by_router_and_shard(tmp_path):
    """Router and shard processes: concurrent requests, prompts longer than a prefill step, a prompt that begins like an
    earlier one; every answer is the greedy continuation of its prompt alone."""
    import os
    import signal
    import subprocess
    import time
    from concurrent.futures import ThreadPoolExecutor

    from test_router_e2e import ROOT, _free_port, _get, _post
    from tgi_b200.router.build import build

    router_bin = build()
    cfg = syn.gisilix_config([A(mlp=dense()), R(mlp=moe()), N(), A(kv_from=0, mlp=dense(40))], width=64, vocab=300)
    sd = syn.gisilix_state_dict(cfg, seed=3)
    path = syn.write_checkpoint(tmp_path / "m", cfg, sd)
    prompts = ["hello world", "a", "the quick brown fox jumps over the lazy dog, twice", "latent", "0123456789" * 4]
    prompts.append(prompts[2][:40] + " and back")
    n = 4
    want = [O.greedy(cfg, sd, [b + 3 for b in p.encode()], n) for p in prompts]
    uds, port = str(tmp_path / "s"), _free_port()
    env = dict(os.environ, PYTHONPATH=ROOT, TGI_B200_CPU_KV_BLOCKS="64", CUDA_VISIBLE_DEVICES="",
               VIRTUAL_ENV=os.environ.get("VIRTUAL_ENV", sys.prefix))
    shard = subprocess.Popen([sys.executable, "-m", "tgi_b200.server.cli", "serve", str(path), "--uds-path", uds,
                              "--dtype", "float32"], env=env, cwd=ROOT)
    router = subprocess.Popen([str(router_bin), "--master-shard-uds-path", uds, "--tokenizer-name", str(path), "--port",
                               str(port), "--hostname", "127.0.0.1", "--max-input-tokens", "64", "--max-total-tokens", "96",
                               "--max-batch-prefill-tokens", "64", "--repo-root", ROOT], env=env, cwd=ROOT)
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
            answers = list(ex.map(ask, prompts[:5])) + [ask(prompts[5])]
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
