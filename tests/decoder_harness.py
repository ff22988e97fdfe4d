"""Helpers of the engine tests of hybrid decoders.  A checkpoint is ``(config, tensors, directory, memo, oracle)`` with
``oracle`` the module of plain reference functions (``forward``, ``greedy``)."""
import random

import pytest
import torch

BACKENDS = ["cpu-f32", pytest.param("cuda-f32", marks=pytest.mark.gpu), pytest.param("cuda-bf16", marks=pytest.mark.gpu)]


@pytest.fixture(params=BACKENDS)
def be(request):
    dev, dt = request.param.split("-")
    return torch.device(dev), torch.float32 if dt == "f32" else torch.bfloat16


def tokens(cfg, n, seed):
    return random.Random(seed).choices(range(cfg["vocab"]), k=n)


def expected(ck, ids):
    cfg, sd, _, memo, oracle = ck
    key = tuple(ids)
    if key not in memo:
        memo[key] = oracle.forward(cfg, sd, ids)
    return memo[key]


def runner_for(ck, be):
    from tgi_b200.models import get_model

    dev, dt = be
    return get_model(str(ck[2]), dtype="float32" if dt == torch.float32 else "bfloat16", device=dev, max_positions=512)


def replay_for(ck, be, max_tokens):
    from tgi_b200.server.replay import Replay

    return Replay(runner_for(ck, be), max_tokens)


def check(got, want, dtype, close_calls=False, normed_blocks=0.0):
    """Per-position error (mean over the vocabulary taken off) against the spread of the expected logits.  ``close_calls``:
    16-bit roundings may tip an expert choice at some position, so a few of them may be further off.  ``normed_blocks``: norms of
    what a block (or a head) returns enlarge 16-bit roundings where it is small, at some positions up to this bound."""
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.std()
    if close_calls and dtype != torch.float32:
        assert err.numel() < 10 or err.quantile(0.75).item() < 0.04, err
        return
    if normed_blocks and dtype != torch.float32:
        assert err.max().item() < normed_blocks and (err.numel() < 30 or err.quantile(0.9).item() < 0.05), err
        return
    assert err.max().item() < (2e-5 if dtype == torch.float32 else 0.04), err


def feed(rp, name, ids, portions, end=True):
    """All logits of ``ids`` brought in ``portions``."""
    out, at = [], 0
    for i, n in enumerate(portions):
        last = at + n == len(ids)
        out.append(rp.step([{"id": name, "tokens": ids[at:at + n], "want": list(range(n))}], [name] if last and end else []))
        at += n
    assert at == len(ids)
    return torch.cat(out)


def requests(prompts, new_tokens):
    from tgi_b200.proto import generate_v3 as pb

    out, block = [], 1
    for i, p in enumerate(prompts):
        r = pb.Request(id=i, inputs="")
        r.parameters.temperature = r.parameters.top_p = r.parameters.typical_p = r.parameters.repetition_penalty = 1.0
        r.stopping_parameters.max_new_tokens = new_tokens[i]
        r.stopping_parameters.ignore_eos_token = True
        n = (len(p) + new_tokens[i] + 15) // 16
        r.blocks.extend(range(block, block + n))
        block += n
        out.append(r)
    return out, block


def generate(runner, prompts, new_tokens, max_prefill=None, late=()):
    """Through ``generate_token``; requests in ``late`` join the running batch after two steps."""
    from tgi_b200.models.flash_causal_lm import FlashCausalLMBatch as B
    from tgi_b200.proto import generate_v3 as pb

    reqs, blocks = requests(prompts, new_tokens)
    runner.init_kv_cache(blocks, state_slots=len(prompts))

    def batch_of(idx):
        return B.from_tokenized(pb.Batch(id=idx[0], requests=[reqs[i] for i in idx], size=len(idx)), [prompts[i] for i in idx],
                                runner.tokenizer, runner.dtype, runner.device)

    early = [i for i in range(len(prompts)) if i not in late]
    batch, toks, step = batch_of(early), {i: [] for i in range(len(prompts))}, 0
    batch.max_prefill_tokens = max_prefill
    while batch is not None:
        if step == 2 and late:
            joined = batch_of(list(late))
            joined.max_prefill_tokens = max_prefill
            batch = B.concatenate([batch, joined])
        gens, batch, _ = runner.generate_token(batch)
        step += 1
        for g in gens:
            toks[g.request_id].extend(g.tokens.token_ids)
        if batch is not None:
            keep = [s.request.id for s in batch.seqs if not s.finished]
            batch = batch.filter(keep)
    return toks


def sure_prompts(ck, count, n, new):
    """Prompts whose greedy continuation never hangs on a near tie."""
    out, seed = [], 100
    while len(out) < count:
        ids = tokens(ck[0], n + 7 * len(out), seed)
        seed += 1
        logits = []
        cur = list(ids)
        for _ in range(new):
            row = ck[4].forward(ck[0], ck[1], cur)[-1]
            logits.append(row)
            cur.append(int(row.argmax()))
        top = torch.stack(logits).topk(2).values
        if (top[:, 0] - top[:, 1]).min() > 0.12:
            out.append((ids, cur[len(ids):]))
    return out
