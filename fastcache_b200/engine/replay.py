"""Replay of given tokens through the engine: teacher-forced steps that return logits instead of sampling.

Every step is one batch of the engine (portions of prompts beside single tokens of other requests), scheduled into
the same blocks and state slots and run by the same prefill and decode steps as generation.
"""
from __future__ import annotations

from contextlib import nullcontext
from typing import Any, Dict, List, Sequence as Seq

import numpy as np
import torch

from ..utils.context import reset_context
from .llm_engine import LLMEngine
from .sequence import Sequence


class TokenReplay:
    def __init__(self, llm: LLMEngine):
        self.llm = llm
        self.live: Dict[str, Sequence] = {}

    @torch.inference_mode()
    def step(self, entries: Seq[Dict[str, Any]], end: Seq[str] = ()) -> torch.Tensor:
        """Feed the next `tokens` of every entry (`id`, `tokens`, `want`) as one batch; returns the logits at the
        wanted places in order, fp32 [wanted, vocab].  The requests named in `end` give back what they hold."""
        sch, runner = self.llm.scheduler, self.llm.model_runner
        pieces = []
        for e in entries:
            if any(not 0 <= w < len(e["tokens"]) for w in e.get("want", ())):
                raise ValueError(f"request {e['id']!r}: a wanted place is not among its {len(e['tokens'])} tokens")
            seq = self.live.get(e["id"])
            if seq is None:
                seq = self.live[e["id"]] = Sequence(e["tokens"])
            pieces.append((seq, list(e["tokens"])))
        logits = torch.empty(0, self.llm.config.hf_config.vocab_size)
        if pieces:
            seqs = sch.schedule_pieces(pieces)
            offsets = np.concatenate([[0], np.cumsum([len(t) for _, t in pieces])])
            rows = [int(o) + int(w) for o, e in zip(offsets, entries) for w in e.get("want", ())]
            stream = torch.cuda.stream(runner.main_stream) if runner.main_stream is not None else nullcontext()
            with stream:
                if all(len(t) == 1 and s.prefill_start > 0 for s, t in pieces):
                    got = runner.run_decode(seqs)[rows]
                else:
                    got = runner.run_prefill(seqs, logits_rows=rows)
                logits = got.float().cpu()
            if runner.main_stream is not None:
                # also when nothing was read back: the next step writes the pinned buffers that this one copies from
                runner.main_stream.synchronize()
            reset_context()
            for s in seqs:
                s.num_computed_tokens, s.prefill_end = s.prefill_end, None
        self.llm.check_device_status()
        for rid in end:
            sch.finish(self.live.pop(rid))
        return logits
