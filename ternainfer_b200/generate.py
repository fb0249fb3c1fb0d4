"""Generation drivers: ``FastGen`` (greedy, whole batches) and ``StepEngine`` (tokens fed request by request).

Both drive any model of ``registry`` through its step interface.  ``FastGen``
mirrors ``generate.py`` of Gu-J/TernaInfer in what matters for the hot path:
the prefill forward and the one-token decode forward are each captured into a
CUDA graph after a warm-up forward (:121-154, :192-224) and replayed with
static input tensors, greedy sampling is an argmax over the logits of each
sequence's last position (:274, :283, :305) - taken inside the output-head
kernel, so the graphs return token ids - and throughput is reported per phase.  Tokenizer, chat format and top-p
sampling of the reference are not rebuilt: prompts are token ids.  ``StepEngine``
keeps a cache per live request, takes the next tokens of a request in portions of
any size and returns logits where they are asked for.
"""
from __future__ import annotations

import argparse
import time
from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from .cache import CachePool, SequenceCache
from .model import ModelArgs, Transformer


def _check_status(model):
    """Models whose kernels report failures on the device raise here."""
    check = getattr(model, "check_status", None)
    if check is not None:
        check()


@dataclass
class GenArgs:
    gen_length: int = 128
    gen_bsz: int = 1
    prompt_length: int = 512
    use_cuda_graph: bool = True


class FastGen:
    def __init__(self, model: Transformer, gen_args: GenArgs, device="cuda"):
        self.model, self.args, self.device = model, gen_args, torch.device(device)
        a = gen_args
        assert a.prompt_length + a.gen_length <= model.max_seq_len
        self.cache = model.make_cache(a.gen_bsz, self.device)
        self._prefill_tokens = torch.zeros((a.gen_bsz, a.prompt_length), dtype=torch.long, device=self.device)
        self._prefill_pos = torch.arange(a.prompt_length, device=self.device)
        self._tokens = torch.zeros((a.gen_bsz, 1), dtype=torch.long, device=self.device)
        self._pos = torch.zeros(1, dtype=torch.long, device=self.device)
        self._prefill_graph = self._decode_graph = None
        self._prefill_next = self._decode_next = None

    @torch.inference_mode()
    def _capture(self):
        s = torch.cuda.Stream()
        s.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(s):          # warm-up forwards outside capture (one-time library set-up)
            self.model(self._prefill_tokens, self.cache, self._prefill_pos, greedy_last=True, start=0)
            self.model(self._tokens, self.cache, self._pos, greedy_last=True)
        torch.cuda.current_stream().wait_stream(s)
        self._prefill_graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(self._prefill_graph):
            self._prefill_next = self.model(self._prefill_tokens, self.cache, self._prefill_pos, greedy_last=True, start=0)
        self._decode_graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(self._decode_graph):
            self._decode_next = self.model(self._tokens, self.cache, self._pos, greedy_last=True)

    @torch.inference_mode()
    def generate(self, prompt: torch.Tensor):
        """prompt [B, prompt_length] token ids -> (tokens [B, gen_length], stats)."""
        a = self.args
        if a.use_cuda_graph and self._decode_graph is None:
            self._capture()
        out = torch.empty((a.gen_bsz, a.gen_length), dtype=torch.long, device=self.device)
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        self._prefill_tokens.copy_(prompt)
        if a.use_cuda_graph:
            self._prefill_graph.replay()
            nxt = self._prefill_next
        else:
            nxt = self.model(self._prefill_tokens, self.cache, self._prefill_pos, greedy_last=True, start=0)
        torch.cuda.synchronize()
        t1 = time.perf_counter()
        for i in range(a.gen_length):
            out[:, i] = nxt
            if i == a.gen_length - 1:
                break
            self._tokens.copy_(nxt[:, None])
            self._pos.fill_(a.prompt_length + i)
            if a.use_cuda_graph:
                self._decode_graph.replay()
                nxt = self._decode_next
            else:
                nxt = self.model(self._tokens, self.cache, self._pos, greedy_last=True)
        torch.cuda.synchronize()
        t2 = time.perf_counter()
        _check_status(self.model)
        stats = {"prefill_s": t1 - t0, "decode_s": t2 - t1,
                 "prefill_tokens_per_s": a.gen_bsz * a.prompt_length / (t1 - t0),
                 "decode_tokens_per_s": a.gen_bsz * (a.gen_length - 1) / (t2 - t1)}
        return out, stats


@dataclass
class _Request:
    cache: SequenceCache
    length: int = 0


class _StepGraph:
    """The one-token forward on one cache, captured once and replayed with static inputs."""

    def __init__(self, model, cache: SequenceCache, device):
        self.tokens = torch.zeros((1, 1), dtype=torch.long, device=device)
        self.pos = torch.zeros(1, dtype=torch.long, device=device)
        self.model, self.cache, self.graph, self.logits = model, cache, None, None

    def run(self, token: int, pos: int) -> torch.Tensor:
        self.tokens.fill_(token)
        self.pos.fill_(pos)
        if self.graph is None:      # the first step runs as it is (library set-up must not be captured)
            logits = self.model(self.tokens, self.cache, self.pos)
            torch.cuda.synchronize()
            self.graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(self.graph):      # records only: the cache advances when it is replayed
                self.logits = self.model(self.tokens, self.cache, self.pos)
            return logits[0]
        self.graph.replay()
        return self.logits[0]


class StepEngine:
    """Feeds requests to a model: ``step`` runs a request's next tokens from what its earlier steps left in its
    cache, ``finish`` gives the cache back.  A step of one token replays a CUDA graph of the decode forward."""

    def __init__(self, model, device="cuda", max_requests: Optional[int] = None, use_cuda_graph: bool = True):
        self.model, self.device, self.use_cuda_graph = model, torch.device(device), use_cuda_graph
        self.pool = CachePool(model, self.device, limit=max_requests)
        self.live: Dict[str, _Request] = {}
        self._graphs: Dict[int, _StepGraph] = {}    # by cache: the pool keeps every cache for good

    @torch.inference_mode()
    def step(self, request: str, tokens: List[int], want: List[int]) -> Optional[torch.Tensor]:
        """fp32 logits [len(want), vocab] at the places ``want`` among these tokens (None if nothing is wanted)."""
        if not tokens or any(not 0 <= t < self.model.vocab_size for t in tokens):
            raise ValueError("a step needs at least one token, all inside the vocabulary")
        if any(not 0 <= w < len(tokens) for w in want):
            raise ValueError("logits wanted outside the step's tokens")
        r = self.live.get(request)
        if (r.length if r else 0) + len(tokens) > self.model.max_seq_len:
            raise ValueError(f"request {request} outgrows the {self.model.max_seq_len} positions of its cache")
        if r is None:
            r = self.live[request] = _Request(self.pool.acquire())
        start, r.length = r.length, r.length + len(tokens)
        if len(tokens) == 1 and self.use_cuda_graph:
            graph = self._graphs.get(id(r.cache))
            if graph is None:
                graph = self._graphs[id(r.cache)] = _StepGraph(self.model, r.cache, self.device)
            logits = graph.run(tokens[0], start)
            if not want:
                return None
            logits = logits.clone()         # the next replay writes the same buffer
            _check_status(self.model)
            return logits
        logits = self.model(torch.tensor([tokens], device=self.device), r.cache,
                            torch.arange(start, r.length, device=self.device),
                            want=torch.tensor(want or [len(tokens) - 1], device=self.device), start=start)
        if not want:
            return None
        _check_status(self.model)
        return logits[0]

    def finish(self, request: str):
        self.pool.release(self.live.pop(request).cache)


def build_random_model(args: ModelArgs, max_seq_len: int, seed: int = 1234, dense: bool = False):
    from .convert.convert_TernaInfer import random_checkpoint
    dic = random_checkpoint(args.dim, args.n_layers, args.n_heads, args.n_kv_heads, args.ffn_dim, args.vocab_size,
                            seed=seed, dense=dense)
    with torch.device("cuda"):
        model = Transformer(args, dic, max_seq_len=max_seq_len)
    return model.cuda().to(torch.bfloat16), dic


def main():
    ap = argparse.ArgumentParser(description="greedy decode of a model folder, or of a random-init BitNet-style model")
    ap.add_argument("--model", default=None, help="folder with config.json and weights; without it: random weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="with --model: number format")
    ap.add_argument("--prompt", default=None, help="token ids with commas between them (otherwise random ids)")
    ap.add_argument("--layers", type=int, default=30)
    ap.add_argument("--bsz", type=int, default=1)
    ap.add_argument("--prompt_length", type=int, default=512)
    ap.add_argument("--gen_length", type=int, default=128)
    ap.add_argument("--no_cuda_graph", action="store_true")
    ap.add_argument("--seed", type=int, default=1234)
    ap.add_argument("--fused_glue", action="store_true", help="fused norm+quantiser kernels, residual add in the epilogue")
    a = ap.parse_args()
    ids = [int(t) for t in a.prompt.split(",")] if a.prompt else None
    if ids:
        a.prompt_length = len(ids)
    if a.model:
        from .registry import load_model
        model = load_model(a.model, getattr(torch, a.dtype), a.prompt_length + a.gen_length)
    else:
        model, _ = build_random_model(ModelArgs(n_layers=a.layers, fused_glue=a.fused_glue), a.prompt_length + a.gen_length,
                                      a.seed)
    gen = FastGen(model, GenArgs(a.gen_length, a.bsz, a.prompt_length, not a.no_cuda_graph))
    if ids:
        if any(not 0 <= t < model.vocab_size for t in ids):
            ap.error("a prompt token lies outside the vocabulary")
        prompt = torch.tensor([ids] * a.bsz, device="cuda")
    else:
        g = torch.Generator(device="cuda").manual_seed(a.seed + 1)
        prompt = torch.randint(0, model.vocab_size, (a.bsz, a.prompt_length), generator=g, device="cuda")
    gen.generate(prompt)            # warm-up (captures the graphs)
    tokens, stats = gen.generate(prompt)
    print({k: round(v, 4) for k, v in stats.items()}, "tokens", tokens[0, :None if ids else 8].tolist())


if __name__ == "__main__":
    main()
