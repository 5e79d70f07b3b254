"""Small hybrid configurations and random checkpoints for the tests, the segment metadata of a hand-made batch, and a
harness that feeds requests through the engine's step and compares every position with an oracle."""

from __future__ import annotations

import contextlib
import copy
import json
import os

import numpy as np
import torch

from oracle import hybrid as hybrid_oracle

MAMBA2 = {"heads": 6, "groups": 3, "state": 24, "vdim": 16, "conv": 4, "norm_groups": 3}
MLSTM = {"heads": 3, "dim": 40, "vdim": 24, "gate_cap": 6.0}
LATENT = {"heads": 5, "dim": 24, "rot_dim": 8, "vdim": 40, "kv_rank": 48, "scale": 0.21,
          "rot": {"base": 5000.0, "dims": 8}, "mask": {"size": 37}}
MIXERS = {"mamba2": MAMBA2, "mlstm": MLSTM, "latent_attention": LATENT}


def layer(kind: str, ff: int | None = 56, **over) -> dict:
    return {"type": kind, "mixer": {**copy.deepcopy(MIXERS[kind]), **over},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def shared(config_layers: list[dict], j: int) -> dict:
    return {**copy.deepcopy(config_layers[j]), "weights_of": j}


def make_config(layers: list[dict], vocab: int = 203, width: int = 88, eps: float = 1e-6) -> dict:
    return {"architecture": "Mapuvik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def default_config() -> dict:
    ls = [layer("latent_attention"), layer("mlstm", ff=None), layer("mamba2", ff=72), layer("latent_attention", ff=40)]
    ls += [shared(ls, 2), shared(ls, 0), shared(ls, 1)]
    return make_config(ls)


def random_checkpoint(config: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    """bf16 tensors by name (what a model folder would hold)."""
    from vllm_metal_b200.lm.hybrid_config import HybridArgs
    from vllm_metal_b200.lm.hybrid_random import random_tensors, tensor_shapes

    args = HybridArgs.parse(config)
    get = random_tensors(args, "cpu", seed)
    return {name: get(name, shape) for name, shape in tensor_shapes(args).items()}


def to_oracle(tensors: dict[str, torch.Tensor]) -> dict[str, np.ndarray]:
    return {k: v.double().numpy() for k, v in tensors.items()}


def write_folder(path, config: dict, tensors: dict[str, torch.Tensor]) -> str:
    from vllm_metal_b200.lm.safetensors_io import save_safetensors

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w", encoding="utf-8") as f:
        json.dump(config, f)
    save_safetensors(os.path.join(path, "model.safetensors"), tensors)
    return str(path)


def make_engine(config: dict, tensors: dict[str, torch.Tensor], dtype=torch.bfloat16, max_tokens: int = 2048,
                max_num_seqs: int = 4, block_size: int = 16, **kw):
    from vllm_metal_b200.lm.registry import family_of
    from vllm_metal_b200.v1.engine import Engine

    family = family_of(config)
    args = family.parse(config)
    model = family.model_class(args)(args, lambda name, shape: tensors[name] if None in shape else tensors[name].reshape(shape),
                                     dtype, "cuda")
    cache = family.make_cache(args, max_tokens // block_size + 1, block_size, max_num_seqs, dtype, "cuda")
    return Engine(model, cache, vocab=args.vocab, max_num_seqs=max_num_seqs, max_model_len=max_tokens, **kw)


def segments(q_lens, context_lens, slots=None, block_size: int = 16, tables=None, device="cuda"):
    """``SegmentMetadata`` of a batch: ``q_lens[i]`` new rows of a request that then holds ``context_lens[i]``."""
    from vllm_metal_b200.attention.context import PagedAttentionContext
    from vllm_metal_b200.attention.impls.segments import segment_metadata

    n = len(q_lens)
    if tables is None:
        tables, at = [], 1
        for c in context_lens:
            k = -(-c // block_size)
            tables.append(list(range(at, at + k)))
            at += k
    cu = [0]
    for q in q_lens:
        cu.append(cu[-1] + q)
    mapping = [tables[i][p // block_size] * block_size + p % block_size
               for i in range(n) for p in range(context_lens[i] - q_lens[i], context_lens[i])]
    ctx = PagedAttentionContext(slot_mapping=mapping, block_tables=tables, context_lens=list(context_lens),
                                offsets=[c - q for c, q in zip(context_lens, q_lens)], cu_seqlens=cu,
                                state_slots=list(slots) if slots is not None else list(range(1, n + 1)))
    return segment_metadata(ctx, block_size, torch.device(device))


@contextlib.contextmanager
def rounded_products(oracle):
    """The oracle with every product's operands and result rounded to 16 bits."""
    def rounded(x):
        return torch.from_numpy(np.ascontiguousarray(x)).bfloat16().double().numpy()

    exact = oracle.linear
    oracle.linear = lambda x, w: rounded(exact(rounded(x), w))
    try:
        yield
    finally:
        oracle.linear = exact


def rounding_error(oracle, config, tensors, tokens, want):
    """How far that rounding alone moves each position's logits: positions where a head's output nearly vanishes before
    its norm are far more sensitive than others."""
    with rounded_products(oracle):
        got = oracle.forward(config, tensors, tokens)
    return np.sqrt(((got - want) ** 2).mean(1)) / max(1.0, want.std())


class Harness:
    """Feeds whole token lists in portions and compares the logits of every position with the oracle's."""

    def __init__(self, config, dtype, seed=0, scale=None, oracle=hybrid_oracle, **kw):
        self.config, self.dtype, self.oracle = config, dtype, oracle
        self.tensors = random_checkpoint(config, seed)
        if scale:
            scale(self.tensors)
        self.oracle_tensors = to_oracle(self.tensors)
        self.engine = make_engine(config, self.tensors, dtype, **kw)
        self.tokens, self.want, self.at, self.limit = {}, {}, {}, {}
        self.positions = self.over = 0

    def request(self, req_id, n, seed=0):
        rng = np.random.default_rng(seed + 100)
        self.tokens[req_id] = rng.integers(0, self.config["vocab"], n).tolist()
        self.want[req_id] = self.oracle.forward(self.config, self.oracle_tensors, self.tokens[req_id])
        self.at[req_id] = 0
        self.limit[req_id] = np.full(n, 4e-5)
        if self.dtype == torch.bfloat16:
            self.limit[req_id] = 1.5e-2 + 3 * rounding_error(self.oracle, self.config, self.oracle_tensors,
                                                             self.tokens[req_id], self.want[req_id])

    def step(self, portions):
        from vllm_metal_b200.v1.engine import StepEntry

        entries, rows, limits = [], [], []
        for req_id, n in portions.items():
            lo = self.at[req_id]
            n = min(n, len(self.tokens[req_id]) - lo)
            if n <= 0:
                continue
            entries.append(StepEntry(req_id, self.tokens[req_id][lo:lo + n], range(n)))
            rows.append(self.want[req_id][lo:lo + n])
            limits.append(self.limit[req_id][lo:lo + n])
            self.at[req_id] += n
        got = self.engine.advance(entries).double().cpu().numpy()
        want = np.concatenate(rows)
        err = np.sqrt(((got - want) ** 2).mean(1)) / max(1.0, want.std())
        ratio = err / np.concatenate(limits)
        # a sensitive position may land on either side of its own estimate; a wrong key or state moves whole stretches
        self.positions += len(ratio)
        self.over += int((ratio > 1).sum())
        allowed = 0 if self.dtype == torch.float32 else max(2, 0.02 * self.positions)
        assert self.over <= allowed and ratio.max() <= 4, (portions, int(ratio.argmax()), float(ratio.max()), self.over)
        for req_id in portions:
            if self.at[req_id] == len(self.tokens[req_id]):
                self.engine.finish(req_id)

    def drain(self, req_id, portions):
        i = 0
        while self.at[req_id] < len(self.tokens[req_id]):
            self.step({req_id: portions[i % len(portions)]})
            i += 1
