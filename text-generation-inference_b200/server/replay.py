"""Replays given token ids through a model, step by step, and writes logits; nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

A step is one JSON line on standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

and is one batch of the engine: every entry brings the next tokens of its request (a portion of a prompt or a
single decoded token), ``want`` lists the tokens whose logits are asked for, ``end`` the requests that give back
what they hold afterwards.  The logits go to ``<out>/<step>.f32`` (little-endian fp32, in the order asked), then
``done <step>`` is printed.

The model, its cache and its step are the serving engine's (``models.get_model``, ``FlashCausalLM.step_logits``).
Pages are taken as requests grow, from a pool of ``--max-tokens`` tokens, so they are used again and again.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Dict, List, Optional

import numpy as np
import torch

LIVE_REQUESTS = 4        # state slots of a replay
EXIT_NO_FLOAT32 = 3


class Replay:
    def __init__(self, runner, max_tokens: int, graphs: bool = True):
        from ..models.flash_causal_lm import BLOCK_SIZE, Seq
        from ..models.state import Pool

        self.runner, self.block = runner, BLOCK_SIZE
        self.pages = Pool(0, -(-max_tokens // BLOCK_SIZE), "KV pages")
        self.live: Dict[str, Seq] = {}
        self._seq, self._next_id = Seq, 0
        runner.init_kv_cache(self.pages.capacity, state_slots=LIVE_REQUESTS)
        if graphs and runner.device.type == "cuda":
            from ..models.graphs import DecodeGraphs

            runner.graphs = DecodeGraphs(runner, self.pages.capacity * BLOCK_SIZE, buckets=[1, 2, LIVE_REQUESTS])
            runner.graphs.capture_all()

    def _admit(self):
        from ..proto import generate_v3 as pb

        self._next_id += 1
        return self._seq(request=pb.Request(id=self._next_id), ids=[], prompt_len=0, cache_len=0, blocks=[],
                         slots=np.zeros(0, dtype=np.int32), stopping=None, top_n=0, prefix_offset=0, read_offset=0)

    def _extend(self, seq, tokens: List[int]):
        seq.ids.extend(tokens)
        seq.prompt_len = len(seq.ids)
        while len(seq.blocks) * self.block < len(seq.ids):
            page = self.pages.take()
            seq.blocks.append(page)
            seq.slots = np.concatenate([seq.slots, np.arange(page * self.block, (page + 1) * self.block, dtype=np.int32)])

    def end(self, name: str):
        seq = self.live.pop(name)
        seq.release_state()
        for page in seq.blocks:
            self.pages.give(page)

    def step(self, entries: List[dict], end: List[str]) -> Optional[torch.Tensor]:
        from ..models.flash_causal_lm import FlashCausalLMBatch

        entries = [e for e in entries if e["tokens"]]
        seqs, counts, want = [], [], []
        for e in entries:
            if e["id"] not in self.live:
                if len(self.live) >= LIVE_REQUESTS:
                    raise RuntimeError(f"more than {LIVE_REQUESTS} live requests")
                self.live[e["id"]] = self._admit()
            seq = self.live[e["id"]]
            self._extend(seq, [int(t) for t in e["tokens"]])
            seqs.append(seq)
            counts.append(len(e["tokens"]))
            want.append([int(w) for w in e.get("want", [])])
        logits = None
        if seqs:
            batch = FlashCausalLMBatch(self._next_id, seqs, None, self.runner.device)
            logits = self.runner.step_logits(batch, counts, want)
            if logits is not None:
                logits = logits.float().cpu()
            elif self.runner.device.type == "cuda":
                torch.cuda.synchronize(self.runner.device)
            if self.runner.device.type == "cuda":
                from ..ops import cuda as K

                code = K.check_status(self.runner.device)
                if code != 0:
                    raise RuntimeError(f"a device-side wait timed out (status {code}); the step's results are invalid")
        for name in end:
            self.end(name)
        return logits


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory the logits are written to")
    ap.add_argument("--max-tokens", required=True, type=int, help="tokens the live requests hold at most")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"],
                    help="cpu: the plain PyTorch ops, for machines without a GPU")
    a = ap.parse_args(argv)
    from ..models import get_model
    from ..models.arch import ARCHS, ModelConfig

    if a.device == "cuda":
        if not torch.cuda.is_available():
            print("trace_run: no CUDA device", file=sys.stderr)
            return 2
        arch = ARCHS.get(ModelConfig.from_path(a.model).model_type)
        if arch is None or not arch.mix:
            if a.dtype == "float32":       # the kernels of the other families are bf16 only
                print("trace_run: this model has no float32 kernels", file=sys.stderr)
                return EXIT_NO_FLOAT32
        else:
            from ..ops import cuda as K

            K.use_kernel_set("decoder")
        device = torch.device("cuda", torch.cuda.current_device())
    else:
        device = torch.device("cpu")
    runner = get_model(a.model, dtype=a.dtype, device=device, max_positions=max(a.max_tokens, 64))
    replay = Replay(runner, a.max_tokens)
    out = Path(a.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        msg = json.loads(line)
        logits = replay.step(msg["entries"], msg.get("end", []))
        if logits is not None:
            part = out / f".{msg['step']}.part"
            part.write_bytes(logits.numpy().astype("<f4").tobytes())
            part.rename(out / f"{msg['step']}.f32")
        print(f"done {msg['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
