"""Sobivik through the engine (loader, caches, scheduler, sampling, replay tool) against ``sobivik_oracle``."""
import io
import json
import random
import sys

import numpy as np
import pytest
import torch

import sobivik_oracle as O
from decoder_harness import (be, check as check_logits, expected, feed, generate, replay_for, requests, runner_for, sure_prompts,  # noqa: F401
                             tokens)
from tgi_b200.utils import synthetic as syn

Ret, Lat, Att, dense = syn.sobivik_retention, syn.sobivik_latent, syn.sobivik_attention, syn.kipedra_dense

CONFIGS = {
    # every mixer twice in other sizes, a layer without a feed-forward in the middle and at the end
    "mixed": syn.sobivik_config([
        Ret(mlp=dense()), Lat(mlp=dense(40)), Att(mlp=dense()), Lat(heads=6, vdim=24, q_rank=24, rot_dim=12, window=37, scaling=None),
        Att(heads=6, kv_heads=3, dim=32, vdim=16, window=33, keep=18, diff=0.6, mlp=dense(56)), Ret(heads=2, dim=40, vdim=48)], eps=2e-2),
    # sizes that are no multiple of 8, other taps and constants
    "odd": syn.sobivik_config([
        Att(heads=3, kv_heads=1, dim=11, vdim=30, window=13, keep=1, diff=0.1, mlp=dense(50)),
        Lat(heads=3, dim=10, vdim=14, q_rank=21, kv_rank=30, rot_dim=6, window=19, base=300.0, mlp=None),
        Ret(heads=3, dim=20, vdim=10, decay=[0.3, 0.9, 1.0], mlp=dense(27))], width=100, vocab=131, eps=1e-3, taps=3, embed_scale=1.0,
        logit_scale=0.3),
    # sizes of the tensor-core kernels; every layer starts or ends a kind
    "wide": syn.sobivik_config([
        Lat(heads=8, dim=128, vdim=128, q_rank=96, kv_rank=512, rot_dim=64, window=70, base=5000.0, scaling=(3.0, 16.0, 1.0, 100), mlp=dense(200)),
        Att(heads=8, kv_heads=2, dim=64, vdim=128, window=40, keep=6, diff=0.5, mlp=dense(128)),
        Ret(heads=4, dim=64, vdim=64, mlp=dense(72)),
        Lat(heads=4, dim=64, vdim=72, q_rank=40, kv_rank=192, rot_dim=32, window=33, mlp=dense(72))], width=128, taps=2, eps=2e-2,
        logit_scale=2.5),
    # no page is ever read
    "recurrent": syn.sobivik_config([Ret(heads=4, dim=64, vdim=24, mlp=dense()), Ret(heads=1, dim=16, vdim=16)], width=64, taps=5,
                                    logit_scale=1.0),
}


# with a small constant in the norms a head's output that nearly vanishes may change its sign with a rounding of 16 bits
BOUNDS = {"mixed": 0.2, "wide": 0.2, "odd": 0.6, "recurrent": 0.6}


def check(got, want, be, name):
    check_logits(got, want, be[1], normed_blocks=BOUNDS[name])


SEEDS = {"mixed": 3, "odd": 1, "wide": 3, "recurrent": 2}
_CKPT = {}


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    def get(name):
        if name not in _CKPT:
            cfg = CONFIGS[name]
            sd = {k: v.to(torch.bfloat16) for k, v in syn.sobivik_state_dict(cfg, seed=SEEDS[name]).items()}
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
    assert rp.pages.available == rp.pages.capacity and rp.runner.state_slots.available == 4


@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_portions_and_decoding(be, checkpoints, expand, name):
    ck = checkpoints(name)
    ids = tokens(ck[0], 150, 1)
    want = expected(ck, ids)
    rp = replay_for(ck, be, 192)
    for portions in ([150], [1] * 150, [2] * 75, [1, 2, 46, 1, 50, 2, 2, 16, 15, 1, 14], [100] + [1] * 50, [47, 3, 60, 40]):
        check(feed(rp, "a", ids, portions), want, be, name)
        free_again(rp)


@pytest.mark.parametrize("name", CONFIGS)
def test_layers_one_by_one(be, checkpoints, name):
    """The stream after every layer, weighted sum included, so that a difference names its layer."""
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
    meta.streams = ops.embed_residual(meta.input_ids, r.model.embed.weight, ck[0]["embedding"]["scale"], len(layers) + 1)
    residual, h = meta.streams[0], None
    for i, (layer, cache) in enumerate(zip(r.model.layer_runs, r.kv_cache)):
        h, residual = layer(h, residual, meta, None, cache)
        assert residual.dtype == torch.float32
        _, after = ops.stream_step(h.out, h.post.weight, residual, layer.norm1.weight, layer.norm1.eps, average=h.average, streams=meta.streams.clone())
        err = (after.double().cpu() - layers[i]).pow(2).mean(-1).sqrt() / layers[i].std()
        if be[1] == torch.float32:
            assert err.max() < 2e-5, (i, err)
        else:
            assert err.max() < BOUNDS[name] and err.quantile(0.9) < 0.04, (i, err)


@pytest.mark.parametrize("name", CONFIGS)
def test_batches_of_unequal_requests(be, checkpoints, expand, name):
    """Up to four live requests in one batch, portions beside single tokens, requests left out of steps, pages and slots
    handed on from finished requests; every logit as if the request were alone."""
    ck = checkpoints(name)
    rp = replay_for(ck, be, 4 * 96)
    rng = random.Random(5)
    waiting = [(f"r{i}", tokens(ck[0], n, 10 + i)) for i, n in enumerate((70, 1, 33, 80, 49, 2, 64, 17, 95))]
    live, seen_pages, seen_slots, gots, wants = {}, [], [], [], []
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
            seen_slots.append(rp.live[n].state.unit)
            rp.end(n)
    check(torch.cat(gots), torch.cat(wants), be, name)
    assert sum(map(len, seen_pages)) > len(set.union(*seen_pages)) and len(seen_slots) > len(set(seen_slots))
    free_again(rp)


def test_first_tokens(be, checkpoints):
    """Nothing comes before a sequence: one- to five-token prompts, alone, on pages and slots that held other requests."""
    for name in ("wide", "mixed"):
        ck = checkpoints(name)
        rp = replay_for(ck, be, 64)
        feed(rp, "old", tokens(ck[0], 33, 8), [33])
        for n in range(1, 6):
            ids = tokens(ck[0], n, 20 + n)
            for portions in ([n], [1] * n):
                check(feed(rp, "a", ids, portions), expected(ck, ids), be, name)


def test_long_decoding(be, checkpoints):
    """Hundreds of single tokens, over many pages, tiles and windows, away from the kept first tokens."""
    ck = checkpoints("wide")
    ids = tokens(ck[0], 330, 9)
    rp = replay_for(ck, be, 384)
    check(feed(rp, "a", ids, [2] + [1] * 328), expected(ck, ids), be, "wide")


def test_state_of_a_request(be, checkpoints):
    """Every layer keeps its last inputs, retention its matrix, the attentions their pages; no prefix is taken over."""
    ck = checkpoints("mixed")
    r = runner_for(ck, be)
    assert r.recurrent and not r.info.use_prefix_caching and r.max_batch_size == 256
    with pytest.raises(ValueError):
        type(r)(r.model, r.tokenizer, r.dtype, r.device, speculate=2)
    r.init_kv_cache(4, state_slots=3)
    for layer, cache in zip(r.model.layer_runs, r.kv_cache):
        assert cache[-1].shape == (3, 3, 80) and cache[-1].dtype == be[1]
        kind = layer.attn.spec.kind
        assert len(cache) == {"decay": 2, "latent": 2, "attention": 3}[kind]
        if kind == "decay":
            assert cache[0].dtype == torch.float32
        if kind == "attention":             # both maps of a key once, values once
            assert cache[0].shape[2] == cache[1].shape[2] == layer.attn.spec.kv_heads


# ---- generation ----------------------------------------------------------------------------------
_SURE = {}


def sure(ck):
    if not _SURE:
        _SURE["wide"] = sure_prompts(ck, 3, 30, 6)
    return _SURE["wide"]


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation(be, checkpoints, graphs):
    ck = checkpoints("wide")
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
    assert runner.overlap_hits == 0          # a step that advances a state runs once


@pytest.mark.gpu
def test_warmup_then_generation(checkpoints, monkeypatch):
    """The server's start: a first step sizes pages and captures the decode steps; generation on them."""
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch as B
    from tgi_b200.proto import generate_v3 as pb

    monkeypatch.setenv("CUDA_MEMORY_FRACTION", "0.1")
    monkeypatch.setenv("CUDA_GRAPHS", "1,2,4")
    ck = checkpoints("wide")
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
    assert cfg.model_type == "sobivik" and cfg.vocab_size == 203
    d = derive_dims(cfg, arch_for(cfg.model_type), 1)
    s = d.mixers
    assert [m.kind for m in s] == ["decay", "latent", "attention", "latent", "attention", "decay"] and all(m.recurrent for m in s)
    assert (d.eps, d.embed_scale, d.logit_scale, d.residual_scale) == (2e-2, 3.0, 1.5, 1.0) and all(m.input_conv == 4 for m in s)
    assert [m.window for m in s] == [0, 24, 20, 37, 33, 0] and [m.keep_first for m in s] == [0, 0, 3, 0, 18, 0]
    assert [m.diff for m in s] == [None, None, 0.3, None, 0.6, None] and s[4].kv_heads == 3 and s[1].kv_heads == 1
    assert [(m.q_rank, m.kv_rank, m.rot_dims) for m in (s[1], s[3])] == [(32, 40, 8), (24, 40, 12)]
    assert s[1].rot_yarn == (4.0, 8.0, 1.0, 128.0) and s[3].rot_yarn is None and s[1].learned_sink and not s[1].rot_interleaved
    assert s[0].k_scale == 24 ** -0.5 and s[5].decay == (0.75, 0.9375) and s[0].qkv_act == "" and s[0].head_norm
    assert [m.feed_forward for m in s] == [True, True, True, False, True, False]
    with pytest.raises(NotImplementedError):
        derive_dims(cfg, arch_for(cfg.model_type), 2)
    for where, value in ((("layers", 0, "type"), "unheard_of"), (("layers", 0, "mlp", "kind"), "unheard_of"), (("layers", 1, "mixer", "rot", "dims"), 4)):
        bad = json.loads(json.dumps(CONFIGS["mixed"]))
        at = bad
        for key in where[:-1]:
            at = at[key]
        at[where[-1]] = value
        with pytest.raises(NotImplementedError):
            ModelConfig(bad)


@pytest.mark.parametrize("name,shape", [("l0.dwa", (3,)), ("l1.canon1", (100, 4)), ("l2.mix.q", None)])
def test_wrong_tensors(tmp_path, name, shape):
    """A sum over the wrong number of results, a convolution of other taps, decays that are not one per head."""
    from tgi_b200.models import get_model

    cfg = json.loads(json.dumps(CONFIGS["odd"]))
    sd = syn.sobivik_state_dict(cfg)
    if shape is None:
        cfg["layers"][2]["mixer"]["decay"].append(0.5)
    else:
        sd[name] = torch.zeros(shape)
    with pytest.raises(ValueError):
        get_model(str(syn.write_checkpoint(tmp_path / "m", cfg, sd)), dtype="float32", device=torch.device("cpu"))


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
    check_logits(got[0], torch.stack([want[10], want[7], want[1]]), torch.float32)
    check_logits(got[1], want[11:], torch.float32)


def test_served_by_router_and_shard(tmp_path):
    """Router and shard processes: more concurrent requests than state slots, prompts longer than a prefill step; every answer
    is the greedy continuation of its prompt alone."""
    import os
    import signal
    import subprocess
    import time
    from concurrent.futures import ThreadPoolExecutor

    from test_router_e2e import ROOT, _free_port, _get, _post
    from tgi_b200.router.build import build

    router_bin = build()
    cfg = syn.sobivik_config([Ret(mlp=dense()), Lat(mlp=dense(40)), Att(mlp=dense())], width=64, vocab=300)
    sd = syn.sobivik_state_dict(cfg, seed=3)
    path = syn.write_checkpoint(tmp_path / "m", cfg, sd)
    prompts = ["hello world", "a", "the quick brown fox jumps over the lazy dog, twice", "retention", "0123456789" * 4]
    prompts.append(prompts[2][:40] + " and back")
    n = 4
    want = [O.greedy(cfg, sd, [b + 3 for b in p.encode()], n) for p in prompts]
    uds, port = str(tmp_path / "s"), _free_port()
    env = dict(os.environ, PYTHONPATH=ROOT, TGI_B200_CPU_KV_BLOCKS="64", CUDA_VISIBLE_DEVICES="", TGI_B200_STATE_SLOTS="2",
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
