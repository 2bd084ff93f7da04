"""Serving side of the library: the registry of model classes, the scheduler, generation.

load_model(folder) reads the folder's config.json and picks the class by its "architecture":
  the decoder architectures of the library (gpt_b200.decoder.Decoder; gptb200_decoder_check_config knows them), and
  "GPT2" (gpt_b200.Model): the seven configuration values beside it and the raw fp32 parameter image in model.bin.

Every class has the same small surface -- open / close a sequence, step over new tokens of sequences, generate -- so that the
scheduler, the command lines and the trace runner serve all of them alike.
"""
from __future__ import annotations

import ctypes
import json
import os
from collections import deque
from dataclasses import dataclass, field

import numpy as np

from .decoder import Decoder


class Gpt2:
    """GPT-2 (gpt_b200.Model) behind the surface of the decoder models: one sequence at a time, its prompt in one step, then token by
    token against the KV cache."""

    batched = False

    def __init__(self, folder: str, config: dict, dtype: str = "float32", device: int = 0, stream: int | None = None):
        import gpt_b200
        if dtype != "float32":
            raise ValueError("GPT2 runs in float32 (3xTF32 products) only")
        self._g = gpt_b200
        self._lib = gpt_b200.load_library()
        self.config = {k: int(config[k]) for k in gpt_b200.CONFIG_KEYS}
        self.model = gpt_b200.Model(self.config, device, stream, use_grad=False)
        path = os.path.join(folder, "model.bin")
        self.model.load_checkpoint(path)
        self.model.set_option("decode_early_launch", 1)
        self.vocab = self.config["vocab_size"]
        self._pitch = self.config["vocab_size_padded"]
        self._ctx = ctypes.c_void_p(self.model.context)
        self._tokens = self._malloc(4 * self.config["max_seq_len"])
        self._logits = self._malloc(4 * self._pitch)
        self._open = None   # (sequence, max_len, length)
        self._count = 0

    def _malloc(self, nbytes: int) -> int:
        p = ctypes.c_void_p()
        rc = self._lib.gptb200_malloc(self._ctx, ctypes.byref(p), nbytes)
        if rc != 0:
            raise self._g.GptB200Error(rc, "gptb200_malloc")
        return int(p.value)

    def close_model(self) -> None:
        if self.model is not None:
            for p in (self._tokens, self._logits):
                self._lib.gptb200_free(self._ctx, ctypes.c_void_p(p))
            self.model.close()
            self.model = None

    def open(self, max_len: int) -> int:
        if self._open is not None:
            raise RuntimeError("GPT2 serves one sequence at a time")
        self._count += 1
        self._open = [self._count, min(max_len, self.config["max_seq_len"]), 0]
        return self._count

    def close(self, seq: int) -> None:
        if self._open is None or self._open[0] != seq:
            raise ValueError(f"sequence {seq} is not open")
        self._open = None

    def length(self, seq: int) -> int:
        return self._open[2] if self._open is not None and self._open[0] == seq else -1

    def _upload(self, tokens) -> None:
        t = np.ascontiguousarray(tokens, np.int32)
        rc = self._lib.gptb200_memcpy_h2d(self._ctx, ctypes.c_void_p(self._tokens), t.ctypes.data_as(ctypes.c_void_p), t.nbytes)
        if rc != 0:
            raise self._g.GptB200Error(rc, "gptb200_memcpy_h2d")

    def _row(self, address: int) -> np.ndarray:
        out = np.empty(self.vocab, np.float32)
        rc = self._lib.gptb200_memcpy_d2h(self._ctx, out.ctypes.data_as(ctypes.c_void_p), ctypes.c_void_p(address), out.nbytes)
        if rc != 0:
            raise self._g.GptB200Error(rc, "gptb200_memcpy_d2h")
        return out

    def step(self, entries, want) -> np.ndarray:
        (seq, tokens), = entries
        if self._open is None or self._open[0] != seq:
            raise ValueError(f"sequence {seq} is not open")
        tokens = np.ascontiguousarray(tokens, np.int32)
        if not len(tokens) or self._open[2] + len(tokens) > self._open[1] or tokens.min() < 0 or tokens.max() >= self.vocab:
            raise ValueError("tokens do not fit the sequence or the vocabulary")
        rows, wanted, first = {}, set(int(w) for w in want), 0
        if self._open[2] == 0:
            self._upload(tokens)
            self.model.generate_begin(self._tokens, 1, len(tokens), self._open[1])
            for w in wanted:
                rows[w] = self._row(self.model.logits_ptr + 4 * self._pitch * w)
            first = len(tokens)
        for i in range(first, len(tokens)):
            self._upload(tokens[i:i + 1])
            self.model.generate_step(self._tokens, self._logits)
            if i in wanted:
                rows[i] = self._row(self._logits)
        self._open[2] += len(tokens)
        self.model.synchronize()
        return np.stack([rows[int(w)] for w in want]) if len(want) else np.empty((0, self.vocab), np.float32)

    def generate(self, seqs, first, steps: int, temperature: float = 0.0, seed: int = 0) -> np.ndarray:
        (seq,), (token,) = seqs, first
        rng, out = np.random.default_rng(seed), np.empty((steps, 1), np.int32)
        for i in range(steps):
            token = sample(self.step([(seq, [token])], [0])[0], temperature, rng)
            out[i, 0] = token
        return out


def _decoder(folder: str, config: dict, dtype: str, device: int, stream: int | None):
    return Decoder(folder, dtype, device, stream)


# architecture name in config.json -> class
REGISTRY = {"Budurax": _decoder, "Lutelorn": _decoder, "GPT2": Gpt2}


def load_model(folder: str, dtype: str = "bfloat16", device: int = 0, stream: int | None = None):
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    name = config.get("architecture")
    if name not in REGISTRY:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(sorted(REGISTRY))})")
    return REGISTRY[name](folder, config, dtype, device, stream)


def sample(logits: np.ndarray, temperature: float, rng) -> int:
    """The largest logit (temperature 0) or a draw from softmax(logits / temperature)."""
    if temperature <= 0.0:
        return int(np.argmax(logits))
    return int(np.argmax(logits.astype(np.float64) / temperature + rng.gumbel(size=logits.shape)))


@dataclass
class Request:
    prompt: list
    max_new_tokens: int
    temperature: float = 0.0
    seed: int = 0
    output: list = field(default_factory=list)
    sequence: int = -1
    fed: int = 0            # tokens of prompt + output that the model has run
    rng: object = None

    @property
    def done(self) -> bool:
        return len(self.output) >= self.max_new_tokens


class Scheduler:
    """Continuous batching: a step takes one token of every request that is generating and fills up with portions of prompts, at
    most `step_tokens` in all; a request leaves as soon as it is done and its slot goes to the next one."""

    def __init__(self, model, max_sequences: int = 8, step_tokens: int = 2048, burst: int = 32):
        self.model = model
        self.max_sequences = max_sequences if model.batched else 1
        self.step_tokens = step_tokens
        self.burst = burst          # longest stretch of steps handed to the model's own generation loop
        self.waiting, self.running = deque(), []

    def submit(self, request: Request) -> Request:
        if not request.prompt:
            raise ValueError("empty prompt")
        request.rng = np.random.default_rng(request.seed)
        self.waiting.append(request)
        return request

    def _admit(self) -> None:
        while self.waiting and len(self.running) < self.max_sequences:
            r = self.waiting.popleft()
            if r.max_new_tokens <= 0:
                continue
            r.sequence = self.model.open(len(r.prompt) + r.max_new_tokens)
            self.running.append(r)

    def _retire(self) -> None:
        for r in [r for r in self.running if r.done]:
            self.model.close(r.sequence)
            r.sequence = -1
            self.running.remove(r)

    def step(self) -> bool:
        """One step; False when nothing is left to do."""
        self._admit()
        if not self.running:
            return False
        # all generating greedily: the model's own loop for a stretch, as far as the request nearest its end goes
        if all(r.output and r.temperature <= 0.0 for r in self.running):
            n = min(self.burst, min(r.max_new_tokens - len(r.output) for r in self.running))
            if n > 1:
                tokens = self.model.generate([r.sequence for r in self.running], [r.output[-1] for r in self.running], n)
                for i, r in enumerate(self.running):
                    r.output += [int(t) for t in tokens[:, i]]
                    r.fed += n
                self._retire()
                return True
        budget, entries, wanted, row = self.step_tokens, [], [], 0
        for r in sorted(self.running, key=lambda r: not r.output):      # those that generate first
            todo = (r.prompt + r.output)[r.fed:]
            take = todo[:budget] if self.model.batched else todo        # GPT2 takes its prompt whole
            if not take:
                continue
            entries.append((r.sequence, take))
            budget -= len(take)
            row += len(take)
            r.fed += len(take)
            if len(take) == len(todo):
                wanted.append((r, row - 1))
        logits = self.model.step(entries, [w for _, w in wanted])
        for (r, _), lg in zip(wanted, logits):
            r.output.append(sample(lg, r.temperature, r.rng))
        self._retire()
        return True

    def run(self) -> None:
        while self.step():
            pass


def generate(model, prompts, max_new_tokens: int, temperature: float = 0.0, seed: int = 0, **scheduler_options):
    """Token lists that continue the prompts (lists of token ids), served together."""
    s = Scheduler(model, **scheduler_options)
    requests = [s.submit(Request(list(p), max_new_tokens, temperature, seed + i)) for i, p in enumerate(prompts)]
    s.run()
    return [r.output for r in requests]
