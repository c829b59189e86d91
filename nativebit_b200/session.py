"""The generation loop every model family shares: one session holds a batch of sequences that advance in lockstep —
their caches, the position, the next token and its logits, all on the device — and runs prompts, portions of prompts
and single decode steps through the model.  The decode step is captured once in a CUDA graph and replayed; the next
token is the arg-max written back into the token buffer, so N steps are N replays without a host round trip.

A model family provides the bodies: `_prefill_body`, `_extend_body`, `_step_body`, and what a step changes besides
position, token and logits (`_step_state`: recurrent states; stale key/value rows past the position are never read)."""
from __future__ import annotations

import torch


class Session:
    def __init__(self, model, batch_size: int, context_len: int, vocab_size: int, device, use_graph: bool = True):
        self.model, self.B, self.context_len = model, batch_size, context_len
        self.dev = device
        self.pos = torch.zeros(1, dtype=torch.long, device=device)
        self.pos_host = 0                     # the same position, tracked on the host: steps past the context are refused
        self.token = torch.zeros(batch_size, 1, dtype=torch.long, device=device)
        self.logits = torch.zeros(batch_size, vocab_size, dtype=torch.float32, device=device)
        self.use_graph = use_graph
        self.graph = None
        self._prefill_graphs = {}             # prompt length -> (captured prefill, its static input)
        self.stream = torch.cuda.Stream(device=device) if torch.device(device).type == "cuda" else None

    # ---- what a model family provides
    def _prefill_body(self, prompt: torch.Tensor) -> None:
        """Runs a whole prompt from an empty cache; leaves self.pos, self.logits and self.token."""
        raise NotImplementedError

    def _extend_body(self, tokens: torch.Tensor, want: list[int]) -> torch.Tensor:
        """Runs tokens (B, T) at positions pos_host ..; returns the logits (B, len(want), V) of those places."""
        raise NotImplementedError

    def _step_body(self) -> None:
        """One token per sequence: consumes self.token, leaves the next one, its logits and the advanced position."""
        raise NotImplementedError

    def _step_state(self) -> list[torch.Tensor]:
        return []

    def _on_reset(self) -> None:
        """Gives back what the finished sequences hold."""

    def check(self) -> None:
        """Raises if a bounded wait inside one of the kernels ever ran out."""

    # ---- the loop
    def reset(self) -> None:
        """Back to an empty sequence: the cache and state of the one before are given back."""
        self.pos.zero_()
        self.pos_host = 0
        self._on_reset()

    @torch.no_grad()
    def prefill(self, prompt: torch.Tensor) -> torch.Tensor:
        """prompt (B, T): fills the caches, sets the position and the first generated token."""
        if prompt.shape[1] > self.context_len:
            raise RuntimeError(f"prompt of {prompt.shape[1]} tokens exceeds the context of {self.context_len}")
        T = int(prompt.shape[1])
        if not self.use_graph or not prompt.is_cuda:
            self._prefill_body(prompt)
        else:
            # one CUDA graph per prompt length: the eager forward is about thirty small launches per layer and
            # is bound by the host; replayed from a graph only the device time remains
            entry = self._prefill_graphs.get(T)
            cur = torch.cuda.current_stream(self.dev)
            if entry is None:
                static_in = prompt.clone()
                self.stream.wait_stream(cur)
                with torch.cuda.stream(self.stream):
                    self._prefill_body(static_in)            # warms every kernel up and IS this call's result
                    self.stream.synchronize()
                    g = torch.cuda.CUDAGraph()
                    with torch.cuda.graph(g, stream=self.stream):
                        self._prefill_body(static_in)
                cur.wait_stream(self.stream)
                self._prefill_graphs[T] = (g, static_in)
            else:
                g, static_in = entry
                static_in.copy_(prompt)
                g.replay()
        self.pos_host = T
        return self.logits

    @torch.no_grad()
    def extend(self, tokens: torch.Tensor, want: list[int] | None = None) -> torch.Tensor:
        """The next tokens (B, T) of the sequences, given by the caller, from the cache and state that earlier calls
        left; returns the logits (B, len(want), V) at the places `want` among them (default: the last).  A single token
        runs as a decode step."""
        T = int(tokens.shape[1])
        want = [T - 1] if want is None else want
        if T < 1 or any(not 0 <= w < T for w in want):
            raise RuntimeError(f"places {want} are not among {T} tokens")
        if self.pos_host + T > self.context_len:
            raise RuntimeError(f"{T} tokens at position {self.pos_host} are past the end of the context ({self.context_len})")
        if T == 1:
            self.token.copy_(tokens)
            self.step()
            return self.logits[:, None, :].expand(-1, len(want), -1)
        out = self._extend_body(tokens, want)
        self.pos_host += T
        self.pos.fill_(self.pos_host)
        return out

    def step(self) -> None:
        """One decode step for every sequence: consumes self.token, leaves the next token there.
        Raises (before anything is launched) when the cache has no free slot left."""
        ctx = self.context_len
        if self.pos_host >= ctx:
            raise RuntimeError(f"decode position {self.pos_host} is past the end of the context ({ctx}): the KV cache is full")
        if not self.use_graph:
            self._step_body()
            self.pos_host += 1
            return
        if self.graph is None:
            # the warm-up and the capture run on the session's stream: it must first see what the caller's
            # stream has written (prefill: caches, position, first token)
            self.stream.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(self.stream):
                changed = [self.pos, self.token, self.logits, *self._step_state()]
                saved = [t.clone() for t in changed]
                for _ in range(min(2, ctx - self.pos_host)):      # warm-up outside capture, inside the context
                    self._step_body()
                self.stream.synchronize()
                for t, s in zip(changed, saved):
                    t.copy_(s)
                self.graph = torch.cuda.CUDAGraph()
                with torch.cuda.graph(self.graph, stream=self.stream):
                    self._step_body()
                # the capture does not execute: state is unchanged; stale cache slots past `pos` are masked
            torch.cuda.current_stream().wait_stream(self.stream)
        self.graph.replay()
        self.pos_host += 1

    @torch.no_grad()
    def generate(self, prompt: torch.Tensor, n_generate: int) -> torch.Tensor:
        """Greedy continuation (B, n_generate) of prompt (B, T)."""
        self.prefill(prompt)
        out = [self.token.clone()]
        for _ in range(n_generate - 1):
            self.step()
            out.append(self.token.clone())
        return torch.cat(out, dim=1)
