"""The step machinery of the single-GPU engines: staging of a decode batch, CUDA-graph capture and replay of a step, the decode
and prefill calls of the runner's interface.

An engine supplies the model: ``_decode_kernels(nb, mode)`` enqueues one decode step on the buffers of ``alloc``,
``_forward_rows(segs)`` runs prompt rows of several sequences, ``_logits(rows)`` turns hidden rows into logits and
``_final_norm(rows)`` normalises them.
"""
from __future__ import annotations

from typing import Sequence

import torch

from ..ops import reference as R


class StepEngine:
    supports_verify = True           # `verify` scores drafted tokens (speculative decoding)
    supports_embeds = True           # prefill takes rows whose input embedding is given
    supports_shift = True            # `shift` drops old positions in place

    def _init_steps(self) -> None:
        self.n_slots = self.n_ctx = 0
        self._graphs: dict[tuple[int, bool], torch.cuda.CUDAGraph] = {}
        self._capture_stream = None
        self.pdl = True
        self.use_graphs = True
        self.launches_per_step = 0
        self.launches_by_key: dict = {}
        self._warm: set = set()
        self._staged = None               # event behind the last copy out of the pinned staging buffer
        self.kernel_launches = 0          # kernels of this library executed so far (graph nodes count individually)
        self.h2d_bytes = self.d2h_bytes = 0

    # -- decode ---------------------------------------------------------------------------------------
    def _run_step(self, nb: int, mode) -> None:
        """mode: False = logits only, True = + arg-max, "loop" = + arg-max and on-device token feedback."""
        key = (nb, mode)
        self.kernel_launches += self.launches_by_key.get(key, 0)
        if not self.use_graphs:
            self._decode_kernels(nb, mode)
            self.launches_by_key[key] = self.launches_per_step
            return
        g = self._graphs.get(key)
        if g is None:
            # the first call runs eagerly (loads the kernels); the second call records the graph
            if key not in self._warm:
                self._warm.add(key)
                self._decode_kernels(nb, mode)
                self.launches_by_key[key] = self.launches_per_step
                return
            g = torch.cuda.CUDAGraph()
            if self._capture_stream is None:      # torch's default capture stream belongs to whichever device captured first
                self._capture_stream = torch.cuda.Stream(device=self.device)
            with torch.cuda.device(self.device), torch.cuda.graph(g, stream=self._capture_stream):
                self._decode_kernels(nb, mode)
            self._graphs[key] = g
        g.replay()

    def _stage(self, slots, tokens, positions) -> int:
        nb = len(slots)
        if nb > self.max_batch:
            raise ValueError(f"decode batch {nb} exceeds {self.max_batch}")
        b = self.buf
        if self._staged is not None:
            self._staged.synchronize()       # the previous step's copy has left the pinned buffer (a caller need not have read its result)
        h = b.host_np
        h[0, :nb] = tokens
        h[1, :nb] = positions
        h[2, :nb] = slots
        b.meta.copy_(b.host_in, non_blocking=True)        # one pinned host -> device copy per step
        if self._staged is None:
            self._staged = torch.cuda.Event()
        self._staged.record()
        self.h2d_bytes += b.host_in.numel() * 4
        return nb

    @torch.no_grad()
    def decode_argmax(self, slots: Sequence[int], tokens: Sequence[int], positions: Sequence[int]) -> list[int]:
        if len(slots) > self.max_batch:      # more sequences than one step takes: consecutive steps
            out: list[int] = []
            for i in range(0, len(slots), self.max_batch):
                j = i + self.max_batch
                out += self.decode_argmax(slots[i:j], tokens[i:j], positions[i:j])
            return out
        nb = self._stage(slots, tokens, positions)
        self._run_step(nb, True)
        self.buf.host_out.copy_(self.buf.sampled, non_blocking=True)
        self.d2h_bytes += self.buf.host_out.numel() * 4
        torch.cuda.current_stream().synchronize()
        return self.buf.host_out_np[:nb].tolist()

    @torch.no_grad()
    def decode(self, slots, tokens, positions) -> torch.Tensor:
        if len(slots) > self.max_batch:
            mb = self.max_batch
            return torch.cat([self.decode(slots[i:i + mb], tokens[i:i + mb], positions[i:i + mb]) for i in range(0, len(slots), mb)])
        nb = self._stage(slots, tokens, positions)
        self._run_step(nb, False)
        return R.softcap(self.buf.logits[:nb].clone(), self.cfg.final_softcap)

    @torch.no_grad()
    def decode_loop(self, slots: Sequence[int], tokens: Sequence[int], positions: Sequence[int], n_steps: int,
                    first_tokens: torch.Tensor | None = None) -> torch.Tensor:
        """Greedy-decode ``n_steps`` tokens for every sequence without leaving the device.

        Returns the sampled ids as an int32 tensor [n_steps, nb] (still on the device).  Used by the
        benchmark's kernel-only measurement and by speculative prefixes where no stop condition can fire.
        """
        if len(slots) > self.max_batch:      # one group of sequences after the other
            parts = []
            for i in range(0, len(slots), self.max_batch):
                j = i + self.max_batch
                parts.append(self.decode_loop(slots[i:j], tokens[i:j], positions[i:j], n_steps,
                                              None if first_tokens is None else first_tokens[i:j]))
            return torch.cat(parts, 1)
        nb = self._stage(slots, tokens, positions)
        if first_tokens is not None:          # ids that are already on the device (e.g. the arg-max of the prefill logits)
            self.buf.tokens[:nb].copy_(first_tokens.to(torch.int32))
        out = torch.empty(n_steps, nb, device=self.device, dtype=torch.int32)
        for i in range(n_steps):
            self._run_step(nb, "loop")
            out[i].copy_(self.buf.sampled[:nb])
        return out

    # -- prefill --------------------------------------------------------------------------------------
    @torch.no_grad()
    def _forward_chunk(self, slot: int, tokens: Sequence[int], pos0: int, x: torch.Tensor | None = None, embeds=None, spans=()) -> torch.Tensor:
        """Chunked prefill: returns the final hidden states [T, d_model] (fp32, before the output norm).

        ``x``: residual stream handed over by the previous pipeline stage (the token ids then only give the chunk length).
        ``embeds`` = (rows, [n, d_model] values): rows whose input embedding is given (image positions); ``spans``: position
        ranges that attend to themselves in both directions.
        """
        return self._forward_rows([(slot, tokens, pos0)], x, embeds, spans)

    @torch.no_grad()
    def prefill_many(self, segs: Sequence[tuple[int, Sequence[int], int]], need_logits: Sequence[bool]) -> list:
        """Prefill chunks of several sequences in one pass (one set of GEMMs over all their rows).  Returns, per chunk, the
        logits after its last token where asked for, else None."""
        x = self._forward_rows(segs)
        ends, at = [], 0
        for _, toks, _ in segs:
            at += len(toks)
            ends.append(at - 1)
        want = [e for e, need in zip(ends, need_logits) if need]
        out: list = [None] * len(segs)
        if want:
            logits = self._logits(x[torch.tensor(want, device=x.device)])
            for j, i in enumerate([i for i, need in enumerate(need_logits) if need]):
                out[i] = logits[j]
        return out

    @torch.no_grad()
    def prefill(self, slot: int, tokens: Sequence[int], pos0: int, need_logits: bool = True, embeds=None, spans=()):
        x = self._forward_chunk(slot, tokens, pos0, embeds=embeds, spans=spans)
        if not need_logits:
            return None
        return self._logits(x[-1:])[0]

    @torch.no_grad()
    def verify(self, slot: int, tokens: Sequence[int], pos0: int) -> torch.Tensor:
        """Logits of every token of the chunk, [T, vocab]: the target-model pass of speculative decoding (one prefill-style
        pass over the drafted tokens instead of one decode step per token)."""
        x = self._forward_chunk(slot, tokens, pos0)
        return self._logits(x)

    @torch.no_grad()
    def hidden(self, slot: int, tokens: Sequence[int]) -> torch.Tensor:
        x = self._forward_chunk(slot, tokens, 0)
        return self._final_norm(x)
