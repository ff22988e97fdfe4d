"""Fuzuvik through the engine (loader, caches, scheduler, sampling, replay tool) against ``fuzuvik_oracle``."""
import io
import json
import random
import sys

import numpy as np
import pytest
import torch

import fuzuvik_oracle as O
from decoder_harness import (be, check, expected, feed, generate, replay_for, requests, runner_for, sure_prompts,  # noqa: F401
                             tokens)
from tgi_b200.utils import synthetic as syn

CONFIGS = {
    # every mixer, shared q/k heads, three layers that mix values (one between them that does not), one without ff
    "mixed": syn.fuzuvik_config([
        syn.fuzuvik_attention(chunk=48, scaling=(4.0, 1.0, 4.0, 128)), syn.fuzuvik_delta(), syn.fuzuvik_lightning(),
        syn.fuzuvik_attention(v_mix=False, heads=6, kv_heads=3, dim=64, vdim=64, chunk=20, rot_dims=40, ff=0),
        syn.fuzuvik_attention(chunk=48, base=300.0), syn.fuzuvik_attention(chunk=100, ff=0)]),
    # recurrent layers first and last, other taps, no shared heads, layers without ff, widths that are no multiple of 8
    "odd": syn.fuzuvik_config([
        syn.fuzuvik_lightning(heads=2, dim=40, vdim=12, ff=0), syn.fuzuvik_delta(heads=3, kv_heads=1, dim=36, vdim=20, conv=2),
        syn.fuzuvik_attention(heads=3, kv_heads=1, dim=20, vdim=52, chunk=33, rot_dims=12, scale=0.4),
        syn.fuzuvik_delta(heads=2, kv_heads=2, dim=16, vdim=16, conv=5, ff=44)], width=100, vocab=131, eps=1e-3, embed_scale=1.0),
    # attention only: head sizes of the tensor-core kernels
    "attention": syn.fuzuvik_config([
        syn.fuzuvik_attention(heads=4, kv_heads=2, dim=128, vdim=128, chunk=64),
        syn.fuzuvik_attention(heads=4, kv_heads=2, dim=128, vdim=128, chunk=37)], width=128),
    # recurrent layers only: no page is ever read
    "recurrent": syn.fuzuvik_config([syn.fuzuvik_delta(heads=4, kv_heads=2, dim=64, vdim=96, conv=3),
                                     syn.fuzuvik_lightning(heads=4, dim=64, vdim=64)], width=64),
}


_CKPT = {}


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    def get(name):
        if name not in _CKPT:
            cfg = CONFIGS[name]
            sd = {k: v.to(torch.bfloat16) for k, v in syn.fuzuvik_state_dict(cfg, seed=len(name)).items()}
            _CKPT[name] = (cfg, sd, syn.write_checkpoint(tmp_path_factory.mktemp(name), cfg, sd), {}, O)
        return _CKPT[name]

    return get


@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_portions_and_decoding(be, checkpoints, name):
    ck = checkpoints(name)
    ids = tokens(ck[0], 150, 1)
    want = expected(ck, ids)
    rp = replay_for(ck, be, 192)
    for portions in ([150], [1] * 150, [2] * 75, [1, 2, 46, 1, 50, 2, 2, 16, 15, 1, 14], [100] + [1] * 50, [47, 3, 60, 40]):
        check(feed(rp, "a", ids, portions), want, be[1])
        assert rp.pages.available == rp.pages.capacity
        assert rp.runner.state_slots is None or rp.runner.state_slots.available == 4


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_layers_one_by_one(be, checkpoints, name):
    """The residual stream after every layer, so that a difference names its layer."""
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch

    ck = checkpoints(name)
    ids = tokens(ck[0], 60, 2)
    layers = []
    O.forward(ck[0], ck[1], ids, layers)
    rp = replay_for(ck, be, 64)
    r = rp.runner
    seq = rp._admit()
    rp._extend(seq, ids)
    meta, _ = r.build_meta(FlashCausalLMBatch(0, [seq], None, r.device), [60], [[0]])
    from tgi_b200 import ops

    residual, h = ops.embed_residual(meta.input_ids, r.model.embed.weight, r.model.dims.embed_scale), None
    for i, layer in enumerate(r.model.layers):
        h, residual = layer(h, residual, meta, None, r.kv_cache[i])
        assert residual.dtype == torch.float32
        err = ((residual + h.float()).double().cpu() - layers[i]).pow(2).mean().sqrt() / layers[i].std()
        assert err < (1e-5 if be[1] == torch.float32 else 0.02), (i, err)


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_batches_of_unequal_requests(be, checkpoints, name):
    """Up to four live requests in one batch, portions beside single tokens, requests left out of steps, pages and slots
    handed on from finished requests; every logit as if the request were alone."""
    ck = checkpoints(name)
    rp = replay_for(ck, be, 4 * 80)
    rng = random.Random(5)
    waiting = [(f"r{i}", tokens(ck[0], n, 10 + i)) for i, n in enumerate((70, 1, 33, 80, 49, 2, 64, 17, 77))]
    live, seen_pages, seen_slots = {}, [], []
    while waiting or live:
        while waiting and len(live) < 4:
            n, ids = waiting.pop(0)
            live[n] = [ids, 0]
        entries, end, wants = [], [], []
        for n, (ids, at) in list(live.items()):
            if rng.random() < 0.2 and len(live) > 1:
                continue
            left = len(ids) - at
            k = min(left, rng.choice([1, 1, 1, 2, 3, 16, 31]))
            entries.append({"id": n, "tokens": ids[at:at + k], "want": list(range(k))})
            wants.append(expected(ck, ids)[at:at + k])
            live[n][1] += k
            if live[n][1] == len(ids):
                end.append(n)
                del live[n]
        if not entries:
            continue
        rng.shuffle(order := list(range(len(entries))))
        got = rp.step([entries[i] for i in order], [])
        check(got, torch.cat([wants[i] for i in order]), be[1])
        for n in end:
            seen_pages.append(set(rp.live[n].blocks))
            seen_slots.append(rp.live[n].state.unit)
            rp.end(n)
    assert len(seen_slots) > len(set(seen_slots)) and set.union(*seen_pages) != set() \
        and sum(map(len, seen_pages)) > len(set.union(*seen_pages))
    assert rp.pages.available == rp.pages.capacity and rp.runner.state_slots.available == 4


def test_first_layer_values_reach_every_later_layer(be, checkpoints):
    """Another first layer value, the same later ones: the change goes through the mixing and nowhere else."""
    cfg, sd, _, _, _ = ck = checkpoints("attention")
    sd2 = dict(sd)
    sd2["l0.mix.o"] = torch.zeros_like(sd["l0.mix.o"])        # the first layer itself writes nothing
    ids = tokens(cfg, 40, 3)
    a = O.forward(cfg, sd2, ids)
    sd2["l1.mix.vmix"] = torch.zeros_like(sd["l1.mix.vmix"])
    b = O.forward(cfg, sd2, ids)
    assert (a - b).abs().max() > 0.1 * a.std()
    check(feed(replay_for(ck, be, 64), "a", ids, [1, 20, 1, 18]), expected(ck, ids), be[1])


# ---- generation ----------------------------------------------------------------------------------
_SURE = {}


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation(be, checkpoints, graphs):
    ck = checkpoints("mixed")
    if "mixed" not in _SURE:
        _SURE["mixed"] = sure_prompts(ck, 3, 30, 6)
    cases = _SURE["mixed"]
    runner = runner_for(ck, be)
    if graphs:
        if be[0].type != "cuda":
            pytest.skip("graphs exist on the GPU only")
        from tgi_b200.models.graphs import DecodeGraphs

    prompts, new = [c[0] for c in cases], [6, 4, 6]

    def run(**kw):
        if graphs:       # captured on the cache that `generate` makes
            init = runner.init_kv_cache

            def init_and_capture(*a, **k):
                init(*a, **k)
                runner.graphs = DecodeGraphs(runner, 96, buckets=[1, 2, 4])
                runner.graphs.capture_all()

            runner.init_kv_cache = init_and_capture
            try:
                return generate(runner, prompts, new, **kw)
            finally:
                runner.init_kv_cache = init
        return generate(runner, prompts, new, **kw)

    want = {i: c[1][:n] for i, (c, n) in enumerate(zip(cases, new))}
    assert run() == want
    assert run(max_prefill=13) == want                      # prompts in portions beside decoded tokens
    assert run(max_prefill=20, late=(1,)) == want
    assert runner.state_slots.available == 3


def test_state_slots_follow_requests(checkpoints):
    """Slots come back when a request finishes, is filtered out, or its batch is dropped; a continued request without its
    state is refused; the shard tells the router how many requests it can hold and that prefixes are not kept."""
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch as B
    from tgi_b200.proto import generate_v3 as pb

    ck = checkpoints("recurrent")
    r = runner_for(ck, (torch.device("cpu"), torch.float32))
    info = r.info
    assert not info.use_prefix_caching and info.support_chunking and info.max_batch_size == r.max_batch_size > 0
    assert not r.overlap_decode
    prompts = [tokens(ck[0], n, n) for n in (9, 12, 5)]
    reqs, blocks = requests(prompts, [4, 4, 4])
    r.init_kv_cache(blocks, state_slots=3)
    make = lambda: B.from_tokenized(pb.Batch(id=0, requests=reqs, size=3), prompts, r.tokenizer, r.dtype, r.device)
    batch = make()
    assert r.state_slots.available == 3
    _, batch, _ = r.generate_token(batch)
    assert r.state_slots.available == 0
    other = make()
    with pytest.raises(RuntimeError, match="recurrent state slots"):
        r.generate_token(other)
    del other
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


# ---- configuration, tool -------------------------------------------------------------------------
def test_config_reader():
    from tgi_b200.models.arch import ModelConfig, arch_for, derive_dims

    cfg = ModelConfig(CONFIGS["mixed"])
    assert cfg.model_type == "fuzuvik" and cfg.vocab_size == 203
    d = derive_dims(cfg, arch_for(cfg.model_type), 1)
    kinds = [s.kind for s in d.mixers]
    assert kinds == ["attention", "delta", "decay", "attention", "attention", "attention"]
    assert d.mixers[0].rot_scaling == (4.0, 1.0, 4.0, 128.0) and d.mixers[4].rot_scaling is None
    assert [s.ff for s in d.mixers] == [96, 96, 96, 0, 96, 0] and not d.mixers[3].v_mix
    assert d.embed_scale == 3.0 and d.eps == 1e-5
    with pytest.raises(NotImplementedError):
        derive_dims(cfg, arch_for(cfg.model_type), 2)
    bad = json.loads(json.dumps(CONFIGS["mixed"]))
    bad["layers"][0]["type"] = "unheard_of"
    with pytest.raises(NotImplementedError):
        ModelConfig(bad)


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


def test_router_reads_the_batch_limit():
    from tgi_b200.proto import generate_v3 as pb

    raw = pb.InfoResponse(max_batch_size=300).SerializeToString()
    assert pb.InfoResponse.FromString(raw).max_batch_size == 300
    assert not pb.InfoResponse().HasField("max_batch_size")


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
    cfg = syn.fuzuvik_config([syn.fuzuvik_attention(chunk=24), syn.fuzuvik_delta(), syn.fuzuvik_lightning(),
                              syn.fuzuvik_attention(chunk=24, ff=0)], width=64, vocab=300)
    sd = syn.fuzuvik_state_dict(cfg, seed=3)
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
