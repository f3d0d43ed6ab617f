"""What every decoder of the framework shares: the loop over a prompt's portions, the decode step
captured as one CUDA graph per token, its position bookkeeping, and greedy generation.

A model class supplies its layers through a handful of hooks:

* `_alloc_caches(batch, length)`       per-layer caches and recurrent state
* `_portion(idx, start)`               hidden rows [B, S, width] of S consecutive tokens, caches advanced
* `_head(hidden)`                      logits of hidden rows
* `_decode_logits(mode)`               logits [B, vocab] of the token in `_tok` at the device position `_pos`
* `_setup_decode_layers`, `_start_decode_layers`, `_release_decode_layers`   decode-time buffers
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch
import torch.nn as nn
from torch import Tensor


def find_multiple(n: int, k: int) -> int:
    return n if n % k == 0 else n + k - (n % k)


class Decoder(nn.Module):
    default_mode = "dense"

    def __init__(self):
        super().__init__()
        self.max_batch_size = self.max_seq_length = -1
        self._graph = None
        self._mode = None

    # -- hooks -----------------------------------------------------------------------------
    @property
    def embedding_table(self) -> Tensor:
        raise NotImplementedError

    def _alloc_caches(self, batch: int, length: int) -> None:
        raise NotImplementedError

    def _portion(self, idx: Tensor, start: int) -> Tensor:
        raise NotImplementedError

    def _head(self, hidden: Tensor) -> Tensor:
        raise NotImplementedError

    def _decode_logits(self, mode: str) -> Tensor:
        raise NotImplementedError

    def _setup_decode_layers(self, batch: int, mode: str) -> None:
        pass

    def _start_decode_layers(self, position: int) -> None:
        pass

    def _release_decode_layers(self) -> None:
        pass

    @property
    def device(self) -> torch.device:
        return self.embedding_table.device

    @property
    def dtype(self) -> torch.dtype:
        return self.embedding_table.dtype

    # -- caches ----------------------------------------------------------------------------
    def setup_caches(self, max_batch_size: int, max_seq_length: int) -> None:
        """Caches for `max_batch_size` sequences of up to `max_seq_length` tokens; kept when they already
        are large enough."""
        if self.max_seq_length >= max_seq_length and self.max_batch_size >= max_batch_size:
            return
        max_seq_length = find_multiple(max_seq_length, 8)
        self.max_seq_length, self.max_batch_size = max_seq_length, max_batch_size
        self._alloc_caches(max_batch_size, max_seq_length)
        self._graph = None

    # -- prefill ---------------------------------------------------------------------------
    @torch.no_grad()
    def forward_portion(self, idx: Tensor, start: int, want: Optional[Sequence[int]] = None) -> Optional[Tensor]:
        """Runs tokens idx [B,S] at positions start.. on the caches that earlier portions left; returns the
        logits [B, len(want), vocab] at the wanted places of the portion (None: of its last token)."""
        B, S = idx.shape
        if B > self.max_batch_size or start < 0 or start + S > self.max_seq_length:
            raise RuntimeError(f"portion of {S} tokens at {start} outside the caches (batch {self.max_batch_size}, "
                               f"max_seq_length={self.max_seq_length})")
        x = self._portion(idx, start)
        if want is None:
            return self._head(x[:, -1:])
        if len(want) == 0:
            return None
        return self._head(x[:, torch.as_tensor(list(want), device=x.device)])

    @torch.no_grad()
    def prefill(self, idx: Tensor, chunk: int = 8192) -> Tensor:
        """idx [B,T] prompt token ids -> logits of the last position [B,vocab].  The prompt is
        processed `chunk` tokens at a time; each portion's queries see everything cached so far."""
        B, T = idx.shape
        assert T <= self.max_seq_length and B <= self.max_batch_size
        for s0 in range(0, T, chunk):
            s1 = min(T, s0 + chunk)
            want = None if s1 == T else ()
            logits = self.forward_portion(idx[:, s0:s1], s0, want)
        return logits[:, -1]

    # -- decode ----------------------------------------------------------------------------
    def _decode_body(self, mode: str) -> None:
        logits = self._decode_logits(mode)
        self._logits = logits
        self._tok.copy_(torch.argmax(logits, dim=-1, keepdim=True))
        self._pos.add_(1)
        self._seqlens.add_(1)

    @torch.no_grad()
    def setup_decode(self, batch: int, mode: Optional[str] = None, use_graph: bool = True) -> None:
        """Allocate the decode-time buffers (current token, position, per-layer staging) and, on a GPU,
        capture one token's work in a CUDA graph."""
        dev = self.device
        mode = self.default_mode if mode is None else mode
        self._mode = mode
        self._tok = torch.zeros(batch, 1, dtype=torch.long, device=dev)
        self._pos = torch.zeros(1, dtype=torch.long, device=dev)
        self._seqlens = torch.zeros(batch, dtype=torch.int32, device=dev)
        self._setup_decode_layers(batch, mode)
        self._graph = None
        self._host_pos = 0
        if use_graph and dev.type == "cuda":
            saved = (self._tok.clone(), self._pos.clone(), self._seqlens.clone())
            side = torch.cuda.Stream(dev)
            side.wait_stream(torch.cuda.current_stream(dev))
            with torch.cuda.stream(side):
                # position 0 of every cache is overwritten by this dry run and by the capture;
                # decoding starts only after `start_decode`, which the caller follows with real tokens
                self._decode_body(mode)
                side.synchronize()
                g = torch.cuda.CUDAGraph()
                with torch.cuda.graph(g, stream=side):
                    self._decode_body(mode)
            torch.cuda.current_stream(dev).wait_stream(side)
            self._graph = g
            self._tok.copy_(saved[0]); self._pos.copy_(saved[1]); self._seqlens.copy_(saved[2])

    def release_decode(self) -> None:
        """Drop the captured graph and the per-layer steps.  Under tensor parallelism call this
        before `torch.distributed.destroy_process_group()`: a live CUDA graph that holds NCCL
        kernels keeps the communicator busy and the teardown waits for it."""
        self._graph = None
        self._release_decode_layers()
        if self.device.type == "cuda":
            torch.cuda.synchronize(self.device)

    @torch.no_grad()
    def start_decode(self, first_token: Tensor, position: int) -> None:
        """`first_token` [B,1] sits at `position` (= number of tokens already cached)."""
        if position >= self.max_seq_length:
            raise RuntimeError(f"start_decode: position {position} outside the caches (max_seq_length="
                               f"{self.max_seq_length})")
        self._host_pos = position                 # host mirror of the device-side position counter
        self._tok.copy_(first_token)
        self._pos.fill_(position)
        self._seqlens.fill_(position)
        self._start_decode_layers(position)

    @torch.no_grad()
    def decode_one_token(self) -> Tensor:
        """Runs one token through the model (greedy); returns the buffer holding the new token.
        Raises before anything is launched when the caches are full (same situation as the
        reference's `_check_input_pos`, GPT-FAST/model.py:279-289, without its device round trip)."""
        if self._host_pos >= self.max_seq_length:
            raise RuntimeError(f"decode position {self._host_pos} outside the caches (max_seq_length="
                               f"{self.max_seq_length}); call setup_caches with a larger length")
        self._host_pos += 1
        if self._graph is not None:
            self._graph.replay()
        else:
            self._decode_body(self._mode)
        return self._tok

    @torch.no_grad()
    def decode_given_token(self, token: Tensor, position: int) -> Tensor:
        """One decode step on a token the caller supplies; returns the buffer holding its logits [B,vocab]."""
        self.start_decode(token, position)
        self.decode_one_token()
        return self._logits


@torch.no_grad()
def generate(model: Decoder, prompt: Tensor, max_new_tokens: int, mode: Optional[str] = None,
             prefill_chunk: int = 8192, use_graph: bool = True, stream_to_host: bool = False):
    """Greedy generation as GPT-FAST/generate.py:246-370: prefill the prompt, take the first new
    token from the prefill logits, then `max_new_tokens - 1` decode steps.  Returns (tokens
    [B, T + max_new_tokens], stats) with `decode_time_s` measured by CUDA events around the decode
    loop and `decode_only_tokens = B * (max_new_tokens - 1)` (generate.py:362-368).  `prompt` may be
    a host tensor; with `stream_to_host` every new token is copied to pinned host memory and waited
    for before the next step is launched (the end-to-end serving pattern)."""
    dev = model.device
    B, T = prompt.shape
    prompt_d = prompt.to(dev, non_blocking=True)
    model.setup_caches(B, T + max_new_tokens + 8)
    cuda = dev.type == "cuda"
    e = [torch.cuda.Event(enable_timing=True) for _ in range(4)] if cuda else None
    # the decode graph's dry run scribbles on cache position 0: capture before the prefill
    model.setup_decode(B, mode, use_graph)
    if cuda:
        e[0].record()
    logits = model.prefill(prompt_d, chunk=prefill_chunk)
    first = torch.argmax(logits, dim=-1, keepdim=True)
    if cuda:
        e[1].record()
    seq = torch.empty(B, T + max_new_tokens, dtype=torch.long, device=dev)
    seq[:, :T] = prompt_d
    seq[:, T] = first[:, 0]
    model.start_decode(first, T)
    host_tok = torch.empty(B, 1, dtype=torch.long).pin_memory() if (cuda and stream_to_host) else None
    if cuda:
        torch.cuda.synchronize(dev)
        e[2].record()
    for i in range(1, max_new_tokens):
        tok = model.decode_one_token()
        seq[:, T + i] = tok[:, 0]
        if host_tok is not None:
            host_tok.copy_(tok, non_blocking=True)
            torch.cuda.current_stream(dev).synchronize()
    stats = {"decode_only_tokens": B * max(0, max_new_tokens - 1)}
    if cuda:
        e[3].record()
        torch.cuda.synchronize(dev)
        stats["prefill_time_s"] = e[0].elapsed_time(e[1]) / 1e3
        stats["decode_time_s"] = e[2].elapsed_time(e[3]) / 1e3
    return seq, stats
