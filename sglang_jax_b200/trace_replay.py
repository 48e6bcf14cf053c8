"""Replay of a recorded batching schedule: given token ids run through a model step by step, the logits at chosen places
are written out, nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

One JSON object per line of standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every entry brings the next tokens of a request (admitted at its first entry); `want` are places among them.  All entries
of a step are one forward batch of the engine: requests with one new token after their first step are decode rows, the
others prefill portions, and a step with both is a mixed batch, built by the scheduler's own `ScheduleBatch`, allocator,
request table and caches and run by the model worker.  `end` lists requests whose pages and state slot are given back
after the step.  A step with wanted places writes `DIR/<step>.f32` (little-endian fp32 `[wanted, vocab]`); after every
step `done <step>` is printed."""

from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


class TraceReplayer:
    """The engine's step machinery without its event loop: at most `max_requests` live requests over a KV pool of
    `max_tokens` token slots."""

    def __init__(self, model_path: str, dtype: str, max_tokens: int, max_requests: int = 4, page_size: int = 64,
                 device: str = "cuda", **server_kw):
        from .configs.model_config import ModelConfig
        from .managers.tp_worker import ModelWorker
        from .mem_cache.memory_pool import ReqToTokenPool
        from .mem_cache.registry import TreeCacheBuildContext, create_tree_cache
        from .models.registry import get_model_class
        from .ops import native
        from .parallel import state as ps
        from .sampling.sampling_params import SamplingParams
        from .server_args import ServerArgs
        max_tokens = -(-max_tokens // page_size) * page_size
        if not ps.get_state().initialized:
            ps.init_distributed(0, 1, device)
        self.sa = ServerArgs(model_path=model_path, dtype=dtype, device=device, page_size=page_size,
                             max_total_tokens=max_tokens, max_running_requests=max_requests,
                             context_length=max_tokens, disable_radix_cache=True, disable_cuda_graph=True,
                             disable_overlap_schedule=True, skip_tokenizer_init=True, **server_kw)
        mc = ModelConfig.from_server_args(self.sa)
        native.prefer_kernel_set(getattr(get_model_class(mc.architectures), "kernel_set", None))
        self.pool = ReqToTokenPool(max_requests, mc.context_len, device, page_size)
        self.worker = ModelWorker(self.sa, mc, req_to_token_pool=self.pool)
        runner = self.worker.model_runner
        built = create_tree_cache(TreeCacheBuildContext(self.sa, mc, self.pool, runner.token_to_kv_pool,
                                                        self.worker.max_total_num_tokens, page_size, None,
                                                        runner.recurrent_pool))
        self.allocator, self.cache = built.allocator, built.tree_cache
        self.vocab, self.page_size = mc.vocab_size, page_size
        self.sampling = SamplingParams(temperature=0.0, max_new_tokens=1 << 30, ignore_eos=True)
        self.reqs: dict = {}

    def _batch(self, reqs):
        from .managers.schedule_batch import ScheduleBatch
        return ScheduleBatch.init_new(reqs, self.pool, self.allocator, self.cache, self.vocab, page_size=self.page_size)

    def step(self, entries: list[dict]) -> np.ndarray:
        """Run one batch; fp32 logits `[wanted, vocab]` in the order of the entries and their `want`."""
        from .managers.schedule_batch import Req
        decode, extend = [], []
        for e in entries:
            req = self.reqs.get(e["id"])
            if req is None:
                req = self.reqs[e["id"]] = Req(e["id"], None, [], self.sampling, vocab_size=self.vocab)
            if req.kv_committed_len and len(e["tokens"]) == 1:
                req.output_ids = list(e["tokens"])            # the token to feed, as if it had just been sampled
                decode.append((req, e))
            else:
                req.origin_input_ids = req.origin_input_ids + list(e["tokens"])
                req.fill_ids = req.origin_input_ids
                extend.append((req, e))
        dec = self._batch([r for r, _ in decode])
        if extend:
            batch = self._batch([r for r, _ in extend])
            batch.prepare_for_extend()
            if decode:
                batch.mix_with_running(dec)
        else:
            batch = dec
            batch.prepare_for_decode()
        wb = batch.get_model_worker_batch()
        order = {e["id"]: i for i, e in enumerate(entries)}
        wanted, at = [], 0                                     # (place in the output, row of the flattened batch)
        for _, e in extend + decode:
            wanted += [((order[e["id"]], k), at + p) for k, p in enumerate(e["want"])]
            at += len(e["tokens"])
        rows = np.asarray([row for _, row in sorted(wanted)], np.int64)
        if extend:
            wb.logits_rows = rows
        res = self.worker.forward_batch_generation(wb, skip_sample=True)
        logits = res.logits_output.next_token_logits
        if not extend:
            import torch
            logits = logits[torch.from_numpy(rows).to(logits.device)]
        for req, _ in extend + decode:
            req.origin_input_ids = req.origin_input_ids + req.output_ids
            req.output_ids = []
            req.fill_ids = req.origin_input_ids
            self.cache.cache_unfinished_req(req)
        return logits.float().cpu().numpy()

    def finish(self, rid: str):
        """Give back what a request holds."""
        req = self.reqs.pop(rid)
        self.cache.cache_finished_req(req, is_insert=False)
        self.pool.free(req.req_pool_idx)


def main(argv=None) -> int:
    p = argparse.ArgumentParser(description="replay a trace of token ids through a model and write logits")
    p.add_argument("--model", required=True)
    p.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    p.add_argument("--out", required=True)
    p.add_argument("--max-tokens", required=True, type=int)
    a = p.parse_args(argv)
    # no kernel choice by timing: it would be measured anew, or read back from an earlier run
    os.environ["SGLB_GEMM_AUTOTUNE"] = "0"
    import torch
    torch.backends.cuda.matmul.allow_tf32 = False
    replay = TraceReplayer(a.model, a.dtype, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"]) if s["entries"] else None
        if logits is not None and any(e["want"] for e in s["entries"]):
            logits.astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        for rid in s["end"]:
            replay.finish(rid)
        print(f"done {s['step']}", flush=True)
    return 0
