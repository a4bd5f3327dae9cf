"""The driver around a decoder: prefill with prefix reuse, the chat loop with stop tokens and usage accounting, and greedy
generation — the methods of the reference's Llama3 class that do not depend on which decoder it drives
(jsgrad/models/llama3.ts:159-164,262-338).
"""
from __future__ import annotations

import time
from dataclasses import dataclass

import numpy as np

from .device import Tensor


@dataclass
class Llama3Usage:
    """jsgrad/models/llama3.ts:159-164."""
    input_tokens: int = 0
    output_tokens: int = 0
    time_to_first_token: float = 0.0
    tokens_per_second: float = 0.0


class Driver:
    """Expects `model` (a decoder.Decoder), `tokenizer`, the sampling settings `temperature`, `top_k`, `top_p`, `alpha_f`,
    `alpha_p`, `max_context`, and the conversation's state `start_pos`, `last_seen_toks`, `usage`."""

    # ---- generation
    def reset(self) -> None:
        self.start_pos, self.last_seen_toks = 0, []

    def _prefill(self, toks, batched: bool = False) -> Tensor | None:
        """Llama3._prefill (jsgrad/models/llama3.ts:298-312).  toks: a list of ids (one conversation) or int32 [B, n].
        At start_pos 0 the part of the prompt that equals what this object saw last is skipped — its K/V rows are
        still in the cache — exactly under the reference's rule: only when one of the two token lists is a prefix of
        the other.  The rest is fed one position per call as the reference does, or, with `batched`, in one
        multi-position forward.  Returns the token picked after the last position fed (None if nothing was fed)."""
        arr = np.asarray(toks, dtype=np.int32)
        if arr.ndim == 1:
            arr = arr[None, :]
        if self.start_pos == 0 and arr.shape[0] == 1:
            cur, last = arr[0].tolist(), list(self.last_seen_toks)
            n = min(len(cur), len(last))
            i = self.model.reusable_prefix(n) if cur[:n] == last[:n] else 0
            self.start_pos += i
            self.last_seen_toks = cur
            arr = arr[:, i:]
        out = None
        if arr.shape[1] == 0:
            return out
        if batched:
            out = self.model.forward(arr, self.start_pos, self.temperature, self.top_k, self.top_p, self.alpha_f, self.alpha_p)
            self.start_pos += arr.shape[1]
            return out
        for i in range(arr.shape[1]):
            out = self.model.call(arr[:, i:i + 1], self.start_pos, self.temperature, self.top_k, self.top_p, self.alpha_f, self.alpha_p)
            self.start_pos += 1
        return out

    def _call(self, tok: int) -> int:
        """One token in, the sampled next token out (Llama3._call, jsgrad/models/llama3.ts:334-337)."""
        res = self.model.call(np.array([[tok]], np.int32), self.start_pos, self.temperature, self.top_k, self.top_p,
                              self.alpha_f, self.alpha_p)
        return int(res.numpy()[0])

    def _system(self, msg: str = "You are an helpful assistant.") -> None:
        """Llama3._system (jsgrad/models/llama3.ts:266-269): begin-of-text + the system turn go through the model."""
        if self.tokenizer is None:
            raise ValueError("no tokenizer: pass tokenizer=Tokenizer.llama(path) (the vocabulary file is not bundled)")
        self._prefill([self.tokenizer.bos_id, *self.tokenizer.encode_message("system", msg)], batched=True)

    def chat(self, messages: list[dict], on_token=None, max_tokens: int | None = None) -> dict:
        """Llama3.chat (jsgrad/models/llama3.ts:270-297): frame the turns, prefill all but the last prompt token, then
        feed tokens back one by one until a stop token comes out.  Returns {'message', 'stop_reason', 'usage'}.  The
        reference loops until a stop token; `max_tokens` and the context length bound the loop here
        (stop_reason 'max_tokens' / 'max_context')."""
        if self.tokenizer is None:
            raise ValueError("no tokenizer: pass tokenizer=Tokenizer.llama(path) (the vocabulary file is not bundled)")
        tk = self.tokenizer
        toks = [t for m in messages for t in tk.encode_message(m["role"], m["content"])] + tk.encode_role("assistant")
        st = time.perf_counter()
        self._prefill(toks[:-1], batched=True)
        usage = Llama3Usage(input_tokens=len(toks) - 1, time_to_first_token=time.perf_counter() - st)
        last_tok, message = toks[-1], {"role": "assistant", "content": ""}
        st = time.perf_counter()
        while True:
            if self.start_pos + 1 > self.max_context:
                return {"message": message, "stop_reason": "max_context", "usage": usage}
            tok = self._call(last_tok)
            self.start_pos += 1
            usage.output_tokens += 1
            usage.tokens_per_second = usage.output_tokens / max(time.perf_counter() - st, 1e-9)
            last_tok = tok
            if tok in tk.stop_tokens:
                return {"message": message, "stop_reason": "end_turn", "usage": usage}
            token = tk.decode([tok])
            message["content"] += token
            if on_token is not None:
                on_token({"message": message, "usage": usage, "token": token})
            if max_tokens is not None and usage.output_tokens >= max_tokens:
                return {"message": message, "stop_reason": "max_tokens", "usage": usage}

    def prefill(self, toks: np.ndarray) -> Tensor:
        """The whole prompt in one multi-position forward (Transformer.forward with S > 1, jsgrad/models/llama.ts:
        201-213) instead of one call per token; returns the greedy token after the last prompt position."""
        out = self.model.forward(np.asarray(toks, dtype=np.int32), self.start_pos, self.temperature, self.top_k, self.top_p,
                                 self.alpha_f, self.alpha_p)
        self.start_pos += toks.shape[1]
        return out

    def generate(self, prompt: np.ndarray, max_new_tokens: int, batched: bool = False) -> np.ndarray:
        """Greedy continuation through the public per-token API: every step copies the token ids to the device, runs
        the (graph-replayed) step and reads the chosen ids back — the `.item()` round trip of the reference's chat
        loop (jsgrad/models/llama3.ts:284-295,334-337).  The prompt goes in one position per call as in the reference, or
        with `batched` in one forward.  prompt: int32 [B, n] -> int32 [B, max_new_tokens]."""
        if self.temperature >= 1e-6:
            raise ValueError("generate() is the greedy loop of the benchmark workloads: construct with temperature=0 "
                             "(sampling runs through chat() / _call())")
        prompt = np.asarray(prompt, dtype=np.int32)
        if prompt.ndim == 1:
            prompt = prompt[None, :]
        B = prompt.shape[0]
        st = time.perf_counter()
        self.last_seen_toks = []  # a seeded workload prompt is always fed whole
        tok = self._prefill(prompt, batched).numpy()
        self.usage.time_to_first_token = time.perf_counter() - st
        out = np.empty((B, max_new_tokens), np.int32)
        st = time.perf_counter()
        for i in range(max_new_tokens):
            out[:, i] = tok
            if i + 1 < max_new_tokens:
                tok = self.model.call_host(tok.reshape(B, 1), self.start_pos)
                self.start_pos += 1
        self.usage.input_tokens, self.usage.output_tokens = int(prompt.size), int(out.size)
        self.usage.tokens_per_second = out.size / max(time.perf_counter() - st, 1e-9)
        return out
