"""Replays given token ids through a rollout engine, step by step, and returns logits.

A trace says which tokens every request feeds at every step; nothing is sampled. The replay goes through the engine the
way generation does: requests enter the C++ scheduler, its plans assign pages and state slots, the plan runs through
``NativeRolloutEngine._forward_plan`` or a captured decode graph, and the scheduler commits one token per sequence —
the trace's next token in place of a sampled one. Useful to compare logits with another implementation, or to follow a
recorded generation exactly.

    engine.initialize(start_loop=False)
    replay = TraceReplay(engine)
    replay.step([TraceEntry("a", [5, 17, 3], [0, 2])])     # logits after its tokens 0 and 2
    replay.step([TraceEntry("a", [8], [0])], end=["a"])
"""

from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np
import torch

_FAR = 1 << 30  # no length limit of its own: a request lives until the trace ends it


@dataclass
class TraceEntry:
    id: str
    tokens: list[int]
    want: list[int] = field(default_factory=list)  # places among ``tokens`` whose logits are asked for


class TraceReplay:
    """One batch at a time: the requests of a step either all start, or all go on by one token."""

    def __init__(self, engine):
        self.e = engine
        # every request runs its own prompt: a request that forks from an equal prompt has no hidden states for it
        engine.sched.set_prompt_sharing(False)
        self.rid: dict[str, int] = {}      # live requests
        self.planned: list[int] = []       # request ids of the last plan, in its order; their next tokens are due

    @torch.no_grad()
    def step(self, entries: list[TraceEntry], end: list[str] = ()) -> torch.Tensor | None:
        """Logits ``[wanted, vocab]`` (fp32, on the host) in the order of ``entries`` and their ``want``; None when
        nothing is wanted. ``end``: requests that give back their pages and slots after this step."""
        s = self.e.sched
        if not entries:
            logits = None
        else:
            fresh = [x for x in entries if x.id not in self.rid]
            if fresh and (len(fresh) != len(entries) or self.rid):
                raise ValueError("a batch has started: its requests go on one token at a time, and no other joins it")
            if fresh:
                hidden, rows = self._start(entries)
            else:
                hidden, rows = self._advance(entries)
            pick = [rows[x.id] + w for x in entries for w in x.want]
            logits = None
            if pick:
                h = hidden.index_select(0, torch.tensor(pick, device=hidden.device))
                logits = self.e.model.logits(h, out_dtype=torch.float32).float().cpu()
        for name in end:
            rid = self.rid.pop(name)
            s.abort(rid)
        self.e._deliver()  # pages were freed by the scheduler; this returns the state slots
        return logits

    def _plan(self, kind: int, expect: int) -> list[int]:
        s = self.e.sched
        got = s.plan()
        if got != kind or s.hdr.n_seqs != expect:
            raise RuntimeError(f"the scheduler planned {s.hdr.n_seqs} requests (kind {got}) instead of {expect} (kind "
                               f"{kind}): the engine's pages, slots or token budget do not hold this batch")
        self.planned = s.seq_ids[:expect].tolist()
        return self.planned

    def _start(self, entries):
        s = self.e.sched
        for x in entries:
            rid = s.add(x.tokens, _FAR, 0, [], True)
            if rid < 0:
                raise ValueError(f"request {x.id}: {len(x.tokens)} tokens do not fit the engine")
            self.rid[x.id] = rid
        order = self._plan(1, len(entries))
        first = {r: int(s.cu[i]) for i, r in enumerate(order)}
        hidden = self.e._forward_plan(1)
        return hidden, {x.id: first[self.rid[x.id]] for x in entries}

    def _advance(self, entries):
        e, s = self.e, self.e.sched
        if any(len(x.tokens) != 1 for x in entries) or {x.id for x in entries} != set(self.rid):
            raise ValueError("every live request goes on by exactly one token")
        nxt = {self.rid[x.id]: x.tokens[0] for x in entries}
        # requests that ended since the plan are gone: the scheduler skips their places
        toks = np.array([nxt.get(r, 0) for r in self.planned], dtype=np.int32)
        if s.commit(toks, np.zeros(len(toks), dtype=np.float32)) < 0:
            raise RuntimeError("the scheduler refused the committed tokens")
        order = self._plan(2, len(entries))
        n = len(order)
        at = {r: i for i, r in enumerate(order)}
        b = e._graphs.bucket(n) if e._graphs is not None else None
        if b is not None:
            e._graphs.run(n, b, s, [0.0] * n, e._rng, e._graph_slots(order))
            hidden = e._graphs.graphs[b][3][:n]
        else:
            hidden = e._forward_plan(2)
        return hidden, {x.id: at[self.rid[x.id]] for x in entries}
