"""What every model of this package shares: one live sequence in a fixed-capacity cache, prompts run in portions,
then one token per step, greedily, the step captured once in a CUDA graph and replayed.

A model supplies the computation:

* `hidden(tokens, pos, end)`: run tokens sitting at the consecutive positions `pos` (device int64) through the
  layers; the cache then holds positions [0, end); returns their hidden states;
* `pick_last(x)`: greedy token after the last of these hidden states (device int64 [1]);
* `logits(x)`: f32 logits of hidden states;
* `_eager_step()`: one token, read from and written to `_tok` at the position in `_pos`, both on the device;
* `step_logits()`: f32 logits [vocab] behind the token the last step picked.

`generate` is the greedy loop (`Qwen3::generate`, llvq-llm/src/model.rs:1041-1073); `feed` appends given tokens to
the live sequence through the same portions and the same step, and returns logits instead of picking.
"""
from __future__ import annotations

from typing import List, Sequence


class TokenLoop:
    PHASES: tuple = ()

    def _init_loop(self, device, capacity: int, prefill_chunk: int) -> None:
        import torch
        if capacity < 1 or prefill_chunk < 1:
            raise ValueError(f"capacity {capacity}, prefill_chunk {prefill_chunk}")
        self.device, self.capacity, self.prefill_chunk = device, capacity, prefill_chunk
        self.positions = torch.arange(capacity, device=device)
        # the token and its position live in fixed device tensors: a captured graph keeps their addresses
        self._tok = torch.zeros(1, dtype=torch.long, device=device)
        self._pos = torch.zeros(1, dtype=torch.long, device=device)
        self._graph = None
        self._only = None   # phase_split: issue only this phase's launches
        self.length = 0     # tokens the live sequence of `feed` holds

    # ---- prompts -----------------------------------------------------------------
    def _portions(self, tokens: Sequence[int], start: int):
        """Run tokens from position `start` on in chunks of `prefill_chunk` (each attends to the cache written so
        far); yields (first index, hidden states) per chunk."""
        import torch
        toks = torch.tensor(list(tokens), device=self.device, dtype=torch.long)
        for lo in range(0, len(tokens), self.prefill_chunk):
            hi = min(len(tokens), lo + self.prefill_chunk)
            yield lo, self.hidden(toks[lo:hi], self.positions[start + lo:start + hi], end=start + hi)

    def prefill(self, prompt: Sequence[int], start: int = 0):
        """Run the prompt through the layers; returns the hidden state of its last token, [1, hidden]."""
        x = None
        for _, x in self._portions(prompt, start):
            pass
        return x[-1:]

    # ---- the greedy loop ---------------------------------------------------------
    def generate(self, prompt: Sequence[int], max_new: int, use_graph: bool = False) -> List[int]:
        """Greedy continuation: prefill, then one token at a time. Takes the cache over from any live sequence."""
        if max_new == 0:
            return []
        n = len(prompt)
        if n == 0:
            raise ValueError("generate: an empty prompt")
        if n + max_new > self.capacity:
            raise ValueError(f"{n} prompt + {max_new} new tokens exceed the cache capacity {self.capacity}")
        self.release()
        nxt = self.pick_last(self.prefill(prompt))
        out = [int(nxt)]
        self.start_decode(nxt, n)
        step = self._graph_step if use_graph else self._eager_step
        while len(out) < max_new:
            step()
            out.append(int(self._tok))  # one scalar read-back per token, as model.rs:1064
        return out

    def start_decode(self, first_token, position: int) -> None:
        """Point the token step at `first_token` (device scalar) sitting at `position` (in place: graph-safe)."""
        self._tok.copy_(first_token.reshape(1))
        self._pos.fill_(position)

    def _graph_step(self) -> None:
        import torch
        if self._graph is None:
            tok0, pos0 = self._tok.clone(), self._pos.clone()
            side = torch.cuda.Stream()
            side.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(side):  # warm-up outside the capture (lazy initialisations)
                self._eager_step()
            torch.cuda.current_stream().wait_stream(side)
            self._tok.copy_(tok0)
            self._pos.copy_(pos0)
            self._graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(self._graph):
                self._eager_step()
            self._tok.copy_(tok0)
            self._pos.copy_(pos0)
        self._graph.replay()

    # ---- given tokens ------------------------------------------------------------
    def release(self) -> None:
        """Give the live sequence's place in the cache back: the next token fed is position 0. Rows left behind are
        never read again, since a position is visible only after its own sequence has written it."""
        self.length = 0

    def feed(self, tokens: Sequence[int], want: Sequence[int] = (), use_graph: bool = True):
        """Append tokens to the live sequence; returns the f32 logits [len(want), vocab] after the places `want`
        among them. One token goes through the token step, more through the prompt path."""
        import torch
        n = len(tokens)
        if n == 0:
            raise ValueError("feed: no tokens")
        if self.length + n > self.capacity:
            raise ValueError(f"{self.length} live + {n} new tokens exceed the cache capacity {self.capacity}")
        if any(not 0 <= w < n for w in want):
            raise ValueError(f"feed: places {list(want)} of {n} tokens")
        rows = {}
        if n == 1:
            self._tok.fill_(int(tokens[0]))
            self._pos.fill_(self.length)
            (self._graph_step if use_graph else self._eager_step)()
            if len(want):
                rows[0] = self.step_logits()
        else:
            for lo, x in self._portions(tokens, self.length):
                here = sorted({w for w in want if lo <= w < lo + x.shape[0]})
                if here:
                    y = self.logits(x[torch.tensor([w - lo for w in here], device=self.device)])
                    rows.update({w: y[k] for k, w in enumerate(here)})
        self.length += n
        return torch.stack([rows[w] for w in want]) if len(want) else None

    # ---- where a token's time goes -----------------------------------------------
    def phase_split(self, reps: int = 10) -> dict:
        """Device time of one token step by phase, in ms: every phase's launches (all layers) captured as a graph
        of their own and replayed `reps` times between two events, at the current position and token. The
        phases run apart here, so their sum leaves out what the whole step gains by overlapping a kernel's
        preamble with its predecessor and adds nothing for the gaps between kernels of different phases. The
        counterpart of the reference's per-phase token timing (llvq-llm/tests/phase_timing.rs). Not for a
        tensor-parallel model under NCCL gathers (a collective inside a partial graph needs every rank)."""
        import warnings
        import torch
        out = {}
        tok0 = self._tok.clone()
        for phase in self.PHASES:
            if phase == "gathers" and not getattr(self, "tp", None):
                continue
            self._only = phase
            try:
                side = torch.cuda.Stream()
                side.wait_stream(torch.cuda.current_stream())
                with torch.cuda.stream(side):
                    self._eager_step()
                torch.cuda.current_stream().wait_stream(side)
                g = torch.cuda.CUDAGraph()
                with warnings.catch_warnings():
                    # a phase whose work the projections' kernels have absorbed captures nothing
                    warnings.filterwarnings("ignore", message="The CUDA Graph is empty")
                    with torch.cuda.graph(g):
                        self._eager_step()
                g.replay()
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                torch.cuda.synchronize()
                e0.record()
                for _ in range(reps):
                    g.replay()
                e1.record()
                torch.cuda.synchronize()
                out[phase] = e0.elapsed_time(e1) / reps
            finally:
                self._only = None
                self._tok.copy_(tok0)
        out["sum"] = sum(out.values())
        return out
