"""Teacher-forced replay: feed given token ids through the engine step by step and write logits.

``bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N`` reads steps from standard input, one
JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` are the requests of the step's batch, each with its next tokens and the places among them whose logits are
wanted; ``end`` names the requests that are finished after the step. The logits of a step go to ``OUT/<step>.f32``
(little-endian fp32 ``[wanted, vocab]`` in the order asked); ``done <step>`` follows on standard output.

The steps run on the serving scheduler's own bookkeeping (request rows, page allocation, step plans) and the engine's
``forward_batch``: prompts' portions and single tokens in one batch take the prefill path, a batch of single tokens the
captured decode graphs."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from .config import SchedulerConfig
from .core import Batch, Req, SamplingParams
from .engine.sample import BatchSamplingArgs
from .scheduler import Scheduler
from .utils import cdiv

MAX_LIVE = 4


class Replayer(Scheduler):
    """A scheduler whose steps are given instead of decided."""

    def __init__(self, config: SchedulerConfig) -> None:
        super().__init__(config)
        self._live: Dict[str, Req] = {}
        self._uids = 0

    def _admit_tokens(self, name: str, ids: torch.Tensor) -> Req:
        if self.table.available_size == 0:
            raise RuntimeError(f"more than {self.config.max_running_req} live requests")
        handle, _ = self.cache.match_req(ids[:0])
        req = Req(input_ids=ids, table_idx=self.table.allocate(), cached_len=0, output_len=0, uid=self._uids,
                  sampling_params=SamplingParams(cache_output=False), cache_handle=handle)
        self.cache.lock(handle)
        self._uids += 1
        self._live[name] = req
        return req

    def step(self, entries: Sequence[Tuple[str, List[int], List[int]]], end: Sequence[str] = ()
             ) -> Optional[torch.Tensor]:
        """``entries``: (request, next tokens, wanted places). Returns the wanted logits ``[wanted, V]`` (CPU fp32)."""
        eng = self.engine
        reqs: List[Req] = []
        uploads = []
        for name, tokens, _ in entries:
            ids = torch.tensor(tokens, dtype=torch.int32)
            req = self._live.get(name)
            if req is None:
                req = self._admit_tokens(name, ids)
            else:
                req.append_host(ids)
                req.cached_len, req.device_len = req.device_len, req.device_len + len(tokens)
            if req.device_len > eng.max_seq_len:
                raise ValueError(f"request {name}: {req.device_len} tokens exceed the limit of {eng.max_seq_len}")
            reqs.append(req)
            uploads.append((req.table_idx, req.cached_len, ids))
        self._upload(uploads)
        result = None
        if reqs:
            decode = all(r.extend_len == 1 and r.cached_len > 0 for r in reqs)
            batch = Batch(reqs=reqs, phase="decode" if decode else "prefill")
            plan = self._make_plan(batch)
            wanted = np.concatenate([plan.cu_q[i] + np.asarray(want, dtype=np.int32)
                                     for i, (_, _, want) in enumerate(entries)]).astype(np.int32)
            # a decode batch keeps one row per request (what its graph computes); nothing is sampled for real:
            # the ids drawn go to the padding request's row of the token pool
            rows = np.arange(len(reqs), dtype=np.int32) if decode else wanted
            plan.sample_rows = rows
            plan.write_idx = np.full(rows.size, self._dummy_slot * self.max_seq_len, dtype=np.int32)
            out = eng.forward_batch(batch, plan, BatchSamplingArgs(), return_logits=True)
            out.wait()
            if wanted.size:
                logits = out.logits[torch.from_numpy(wanted).long().to(out.logits.device)] if decode else out.logits
                result = eng.sampler.condition_logits(logits, BatchSamplingArgs()).float().cpu()
        for name in end:
            req = self._live.pop(name)
            req.cached_len = req.device_len
            self._free_req_resources(req, insert=False)
        return result

    def _upload(self, uploads) -> None:
        pool = self.engine.token_pool
        if pool.is_cuda:
            with torch.cuda.stream(self.engine.stream):
                for slot, at, ids in uploads:
                    pool[slot, at:at + ids.numel()].copy_(ids)
        else:
            for slot, at, ids in uploads:
                pool[slot, at:at + ids.numel()].copy_(ids)


def make_replayer(model: str, dtype: str, max_tokens: int, device: str = "cuda", page_size: int = 16) -> Replayer:
    return Replayer(SchedulerConfig(
        model_path=model, dtype=dtype, device=device, page_size=page_size, num_page_override=cdiv(max_tokens, page_size),
        max_running_req=MAX_LIVE, max_extend_tokens=max_tokens, cache_type="naive", offline_mode=True))


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", choices=("cuda", "cpu"), default="cuda", help="cpu: the reference ops, for debugging")
    ap.add_argument("--page-size", type=int, default=16)
    args = ap.parse_args(argv)
    done = os.fdopen(os.dup(1), "w")       # answers; whatever else prints goes to standard error
    os.dup2(2, 1)
    from .models.config import ModelConfig

    mc = ModelConfig.from_hf(args.model)
    if args.dtype == "float32" and args.device == "cuda" and not mc.has_fp32_kernels:
        print(f"trace_run: {mc.model_type} has no 32-bit kernels", file=sys.stderr)
        return 3
    if args.device == "cuda":
        from . import build
        from .ops import _lib

        if not os.path.exists(_lib.LIB_PATH):
            if mc.has_fp32_kernels:
                part = ("pair" if mc.depth_average else "heads" if mc.layered else "layered" if mc.layer_specs
                        else "latent")
                _lib.use_part(build.build_cuda(part=part))
            else:
                build.build_cuda()
    torch.backends.cuda.matmul.allow_tf32 = False
    rep = make_replayer(args.model, args.dtype, args.max_tokens, args.device, args.page_size)
    for line in sys.stdin:
        if not line.strip():
            continue
        msg = json.loads(line)
        logits = rep.step([(e["id"], e["tokens"], e.get("want", [])) for e in msg["entries"]], msg.get("end", []))
        if logits is not None:
            logits.numpy().astype("<f4").tofile(os.path.join(args.out, f"{msg['step']}.f32"))
        print(f"done {msg['step']}", file=done, flush=True)
    rep.engine.shutdown()
    return 0
