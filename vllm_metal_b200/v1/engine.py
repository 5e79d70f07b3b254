"""Self-contained engine over ``PagedModelRunner``: page and state-slot allocation, continuous batching with chunked
prefill, greedy sampling.  It serves every model family of ``lm/registry.py`` without vLLM's scheduler (under vLLM the
same runner is driven by ``v1/worker.py``); ``generate`` is its entry point, ``advance`` the step underneath -- feed
given tokens to live requests, get logits -- which a trace replay uses directly.

Pages and slots are handed out here and nowhere else; admission reserves what a request can grow to, so a running
request never has to be evicted."""

from __future__ import annotations

from collections import deque
from collections.abc import Sequence
from dataclasses import dataclass, field

import torch

from ..attention.caches.state_cache import StateSlots
from ..lm.registry import family_of, read_config
from .model_runner import PagedModelRunner

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class BlockPool:
    """Page ids 1..n (page 0 is the padding target of every pool)."""

    def __init__(self, num_blocks: int, block_size: int) -> None:
        self.num_blocks, self.block_size = num_blocks, block_size
        self._free = list(range(num_blocks, 0, -1))

    @property
    def num_free(self) -> int:
        return len(self._free)

    def blocks_for(self, tokens: int) -> int:
        return -(-tokens // self.block_size)

    def extend(self, blocks: list[int], tokens: int) -> None:
        """Grow a request's page list to hold ``tokens`` tokens."""
        need = self.blocks_for(tokens) - len(blocks)
        if need > len(self._free):
            raise RuntimeError(f"{need} more pages wanted, {len(self._free)} free")
        for _ in range(need):
            blocks.append(self._free.pop())

    def release(self, blocks: list[int]) -> None:
        self._free.extend(reversed(blocks))
        blocks.clear()


@dataclass
class Request:
    req_id: str
    tokens: list[int] = field(default_factory=list)   # prompt and generated tokens
    prompt_len: int = 0
    max_new_tokens: int = 0
    stop_token: int | None = None
    num_computed: int = 0
    blocks: list[int] = field(default_factory=list)

    @property
    def reserve(self) -> int:
        return self.prompt_len + self.max_new_tokens

    @property
    def output(self) -> list[int]:
        return self.tokens[self.prompt_len:]


@dataclass
class StepEntry:
    """``tokens`` appended to request ``req_id``; logits wanted after the tokens at ``want``."""

    req_id: str
    tokens: Sequence[int]
    want: Sequence[int] = ()


class Engine:
    def __init__(self, model, cache, *, vocab: int, max_num_seqs: int, max_model_len: int,
                 max_batched_tokens: int = 2048, use_cuda_graph: bool = True) -> None:
        self.model, self.cache, self.vocab = model, cache, vocab
        self.max_num_seqs, self.max_model_len = max_num_seqs, max_model_len
        self.max_batched_tokens = max(max_batched_tokens, max_num_seqs)
        self.pool = BlockPool(cache.num_blocks - 1, cache.block_size)
        self.slots = StateSlots(max_num_seqs)
        self.runner = PagedModelRunner(model, cache, max_batch=max_num_seqs, max_model_len=max_model_len,
                                       use_cuda_graph=use_cuda_graph)
        self.live: dict[str, Request] = {}
        self.waiting: deque[Request] = deque()

    @classmethod
    def from_folder(cls, folder: str, *, dtype: str = "bfloat16", max_tokens: int = 8192, max_num_seqs: int = 64,
                    max_model_len: int | None = None, block_size: int = 16, device: str = "cuda", **kw) -> Engine:
        """``max_tokens``: what the pool holds at any time, over all requests."""
        config = read_config(folder)
        family = family_of(config)
        torch_dtype = DTYPES[dtype]
        if torch_dtype not in family.dtypes:
            raise NotImplementedError(f"family '{family.name}' does not run in {dtype}")
        args = family.parse(config)
        model = family.load(args, folder, torch_dtype, device)
        blocks = -(-max_tokens // block_size) + 1
        cache = family.make_cache(args, blocks, block_size, max_num_seqs, torch_dtype, device)
        return cls(model, cache, vocab=family.vocab(args), max_num_seqs=max_num_seqs,
                   max_model_len=max_model_len or max_tokens, **kw)

    # -- the step ------------------------------------------------------------------------------
    def _request(self, req_id: str) -> Request:
        if req_id not in self.live:
            if len(self.live) >= self.max_num_seqs:
                raise RuntimeError(f"{self.max_num_seqs} requests are live already")
            self.live[req_id] = Request(req_id)
        return self.live[req_id]

    def _run(self, work: list[tuple[Request, int]], want: list[list[int]] | None) -> torch.Tensor:
        """Compute the next ``n`` tokens of every request as one batch.  Logits, in the order of ``work``: of each
        request's last token (``want`` None) or of the places listed."""
        for req, n in work:
            self.pool.extend(req.blocks, req.num_computed + n)
        slot = {req.req_id: self.slots.acquire(req.req_id) for req, _ in work} if self.runner.stateful else None
        decode = [i for i, (req, n) in enumerate(work) if n == 1 and req.num_computed > 0]
        prefill = [i for i in range(len(work)) if i not in set(decode)]
        order = decode + prefill
        ids: list[int] = []
        first: dict[int, int] = {}
        for i in order:
            req, n = work[i]
            first[i] = len(ids)
            ids.extend(req.tokens[req.num_computed:req.num_computed + n])
        slots = None if slot is None else [slot[work[i][0].req_id] for i in order]
        rows = [first[i] + k for i, (_, n) in enumerate(work) for k in (want[i] if want is not None else [n - 1])]
        r = self.runner
        if not prefill and r.use_cuda_graph and len(decode) <= r.max_batch:
            # pure decode: pinned staging -> one H2D -> graph replay
            r.decode_step(ids, [work[i][0].blocks for i in order], [work[i][0].num_computed for i in order],
                          state_slots=slots, sync=False)
            logits = r.last_logits[rows] if rows else r.last_logits[:0]
            torch.cuda.current_stream().synchronize()  # the pinned mirrors are free for the next step
        else:
            dec = [(work[i][0].blocks, work[i][0].num_computed) for i in decode]
            pre = [(work[i][0].blocks, work[i][1], work[i][0].num_computed) for i in prefill]
            logits = r.forward_rows(ids, dec, pre, rows, slots)
        for req, n in work:
            req.num_computed += n
        return logits

    def advance(self, entries: Sequence[StepEntry]) -> torch.Tensor:
        """Append the entries' tokens to their requests (admitting new ones) and compute them as one batch; logits
        ``[wanted, vocab]`` in the order of the entries and of their ``want``."""
        work, want = [], []
        for e in entries:
            if not e.tokens:
                raise ValueError(f"request {e.req_id}: no tokens")
            if any(not 0 <= t < self.vocab for t in e.tokens):
                raise ValueError(f"request {e.req_id}: token outside the vocabulary of {self.vocab}")
            if any(not 0 <= k < len(e.tokens) for k in e.want):
                raise ValueError(f"request {e.req_id}: wanted place outside its {len(e.tokens)} tokens")
            req = self._request(e.req_id)
            if req.num_computed + len(e.tokens) > self.max_model_len:
                raise ValueError(f"request {e.req_id}: longer than {self.max_model_len} tokens")
            req.tokens.extend(e.tokens)
            work.append((req, len(e.tokens)))
            want.append(list(e.want))
        if len({req.req_id for req, _ in work}) != len(work):
            raise ValueError("a request appears twice in one step")
        if not work:
            return torch.empty((0, self.vocab), dtype=torch.float32, device=self.cache.device)
        return self._run(work, want)

    def finish(self, req_id: str) -> None:
        """Give back what a request holds."""
        req = self.live.pop(req_id, None)
        if req is not None:
            self.pool.release(req.blocks)
        self.slots.release(req_id)

    # -- scheduling and generation -----------------------------------------------------------------
    def add_request(self, req_id: str, prompt: Sequence[int], max_new_tokens: int, stop_token: int | None = None) -> None:
        req = Request(req_id, list(prompt), len(prompt), max_new_tokens, stop_token)
        if not prompt or max_new_tokens < 1:
            raise ValueError(f"request {req_id}: needs a prompt and at least one token to generate")
        if any(not 0 <= t < self.vocab for t in prompt):
            raise ValueError(f"request {req_id}: token outside the vocabulary of {self.vocab}")
        if req_id in self.live or any(r.req_id == req_id for r in self.waiting):
            raise ValueError(f"request {req_id} exists already")
        if req.reserve > self.max_model_len or self.pool.blocks_for(req.reserve) > self.pool.num_blocks:
            raise ValueError(f"request {req_id}: {req.reserve} tokens never fit")
        self.waiting.append(req)

    def schedule(self) -> list[tuple[Request, int]]:
        """Decoding requests first, one token each, then prompt portions into what is left of the token budget; new
        requests are admitted while their whole length is covered by free, unpromised pages."""
        work, budget = [], self.max_batched_tokens
        for req in self.live.values():
            if req.num_computed + 1 == len(req.tokens) and req.num_computed >= req.prompt_len:
                work.append((req, 1))
                budget -= 1
        for req in self.live.values():
            n = min(budget, req.prompt_len - req.num_computed)
            if n > 0:
                work.append((req, n))
                budget -= n
        promised = sum(self.pool.blocks_for(r.reserve) - len(r.blocks) for r in self.live.values())
        while self.waiting and budget > 0 and len(self.live) < self.max_num_seqs:
            req = self.waiting[0]
            need = self.pool.blocks_for(req.reserve)
            if promised + need > self.pool.num_free:
                break
            promised += need
            self.waiting.popleft()
            self.live[req.req_id] = req
            n = min(budget, req.prompt_len)
            work.append((req, n))
            budget -= n
        return work

    def step(self) -> list[Request]:
        """One scheduled batch; returns the requests it finished."""
        work = self.schedule()
        if not work:
            return []
        done: list[Request] = []
        tokens = self.runner._greedy(self._run(work, None)).tolist()
        for (req, _), token in zip(work, tokens, strict=True):
            if req.num_computed < len(req.tokens):
                continue  # a portion that does not reach the end of the prompt samples nothing
            req.tokens.append(int(token))
            if len(req.output) >= req.max_new_tokens or token == req.stop_token:
                done.append(req)
        for req in done:
            self.finish(req.req_id)
        return done

    def generate(self, prompts: Sequence[Sequence[int]], max_new_tokens: int, stop_token: int | None = None) -> list[list[int]]:
        """Greedy continuations of ``prompts``."""
        for i, p in enumerate(prompts):
            self.add_request(str(i), p, max_new_tokens, stop_token)
        outputs: dict[str, list[int]] = {}
        while self.live or self.waiting:
            for req in self.step():
                outputs[req.req_id] = req.output
        return [outputs[str(i)] for i in range(len(prompts))]


__all__ = ["BlockPool", "Engine", "Request", "StepEntry"]
