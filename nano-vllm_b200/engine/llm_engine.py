"""Generation over token ids: add requests, step, collect (the surface of nanovllm/engine/llm_engine.py:16-93 without
its tokenizer and worker processes)."""
from __future__ import annotations

import os
from dataclasses import dataclass

import torch.distributed as dist

from ..models.registry import config_from_dict, load_config
from ..utils.loader import Checkpoint
from .cache_manager import CacheManager
from .model_runner import ModelRunner, Seq
from .scheduler import Scheduler


@dataclass
class SamplingParams:
    """temperature 0 = greedy."""
    temperature: float = 0.0
    max_tokens: int = 64
    ignore_eos: bool = False


def ensure_process_group() -> None:
    """The layers read rank and world size from torch.distributed; a single process makes a group of its own."""
    if not dist.is_initialized():
        dist.init_process_group("gloo", store=dist.HashStore(), rank=0, world_size=1)


class LLMEngine:

    def __init__(self, model, weights=None, **runner_args):
        """model: a folder with config.json and *.safetensors, a config dict, or a config object (then `weights` maps
        checkpoint names to tensors; without it the weights are random)."""
        ensure_process_group()
        if isinstance(model, (str, os.PathLike)):
            config = load_config(model)
            weights = Checkpoint(model) if weights is None else weights
        else:
            config = config_from_dict(model) if isinstance(model, dict) else model
        self.config = config
        self.runner = ModelRunner(config, full_weights=weights, **runner_args)
        r = self.runner
        self.cache = CacheManager(r.num_kvcache_blocks, r.block_size, r.num_state_slots)
        self.scheduler = Scheduler(self.cache, r.max_num_seqs, r.max_num_batched_tokens)
        self._params: dict[int, SamplingParams] = {}
        self._prompt_len: dict[int, int] = {}

    def add_request(self, prompt: list[int], params: SamplingParams) -> Seq:
        if not prompt:
            raise ValueError("empty prompt")
        if len(prompt) + params.max_tokens > self.runner.max_model_len:
            raise ValueError(f"{len(prompt)} prompt + {params.max_tokens} new tokens exceed max_model_len={self.runner.max_model_len}")
        seq = Seq(list(prompt))
        self._params[id(seq)], self._prompt_len[id(seq)] = params, len(prompt)
        self.scheduler.add(seq)
        return seq

    def step(self) -> list[Seq]:
        """One prefill or decode step; returns the sequences that finished in it."""
        seqs, counts = self.scheduler.schedule()
        if not seqs:
            return []
        temps = [self._params[id(s)].temperature for s in seqs]
        greedy = all(t <= 0 for t in temps)
        temperatures = None if greedy else [max(t, 1e-5) for t in temps]
        tokens = self.runner.step(seqs, counts is not None, temperatures, num_new=counts)
        finished = []
        for i, (s, t) in enumerate(zip(seqs, tokens)):
            if counts is not None and not self.scheduler.prefilled(s, counts[i]):
                continue
            s.num_cached_tokens = len(s)
            s.token_ids.append(t)
            p = self._params[id(s)]
            stop = not p.ignore_eos and self.config.eos_token_id is not None and t == self.config.eos_token_id
            if stop or len(s) - self._prompt_len[id(s)] >= p.max_tokens:
                self.scheduler.finish(s)
                finished.append(s)
        return finished

    def generate(self, prompts: list[list[int]], params: SamplingParams | list[SamplingParams]) -> list[list[int]]:
        if not isinstance(params, list):
            params = [params] * len(prompts)
        seqs = [self.add_request(p, sp) for p, sp in zip(prompts, params)]
        while not self.scheduler.done():
            self.step()
        out = [s.token_ids[self._prompt_len[id(s)]:] for s in seqs]
        for s in seqs:
            del self._params[id(s)], self._prompt_len[id(s)]
        return out

    def exit(self) -> None:
        self.runner.exit()


LLM = LLMEngine
