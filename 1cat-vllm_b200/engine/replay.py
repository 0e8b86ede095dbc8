"""Trace replay: given token ids run through the engine step by step and selected logits come back; nothing is sampled.

The engine is the one that generates (executor, worker, runner, paged cache and its manager): only the choice of each step's tokens and
the sampling are replaced. A step names requests and their next tokens; all of them run as one batch, portions of prompts beside single
tokens, over whatever earlier steps left in the cache."""
from __future__ import annotations

from typing import Optional

from onecat_vllm.config import EngineArgs
from onecat_vllm.engine.core import EngineCore
from onecat_vllm.request import Request, RequestStatus


class TraceReplay:
    def __init__(self, model: str, dtype: str, max_tokens: int, max_live: int = 4, device: str = "auto", block_size: int = 16, **engine_args):
        """``max_tokens``: the most tokens that live requests hold at any time; the cache pool is made for them."""
        max_tokens = -(-max_tokens // block_size) * block_size
        args = EngineArgs(model=model, dtype=dtype, device=device, block_size=block_size, max_model_len=max_tokens, max_num_batched_tokens=max_tokens,
                          max_num_seqs=max_live, num_gpu_blocks_override=max_tokens // block_size + 1, kv_cache_memory_bytes=1 << 30,
                          enable_prefix_caching=False, async_scheduling=False, **engine_args)   # a step runs exactly the tokens it brings
        self.core = EngineCore(args.create_engine_config(), log_stats=False)

    def step(self, entries: list[dict], end: list[str] = ()) -> Optional["torch.Tensor"]:
        """``entries``: ``{"id", "tokens", "want"}`` per request, ``want`` being offsets among its tokens. Returns the wanted logits (fp32,
        on the host, in the order of the entries and of ``want``) or None; ``end`` names the requests that are finished afterwards."""
        sch = self.core.scheduler
        counts: dict = {}
        for e in entries:
            rid, toks = e["id"], [int(t) for t in e["tokens"]]
            bad = next((t for t in toks if not 0 <= t < self.core.cfg.model_config.vocab_size), None)
            if bad is not None:
                raise ValueError(f"token {bad} of request {rid} is outside the vocabulary")
            if any(not 0 <= j < len(toks) for j in e.get("want") or ()):
                raise ValueError(f"request {rid} asks for logits outside its {len(toks)} tokens")
            if rid in counts:
                raise ValueError(f"request {rid} appears twice in one step")
            if not toks:
                continue
            counts[rid] = len(toks)
            if rid in sch.requests:
                sch.requests[rid].append_output_token_ids(toks)
            else:
                sch.add_request(Request(rid, toks, None))
        logits = None
        if counts:
            so = sch.schedule_exact(counts)
            so.logits_for = {e["id"]: list(e.get("want") or ()) for e in entries if e["id"] in counts}
            logits = self.core._guarded(so, lambda: self.core.executor.execute_model(so)).logits
        if end:
            sch.finish_requests([r for r in end], RequestStatus.FINISHED_ABORTED)
        return logits

    def close(self) -> None:
        self.core.shutdown()
