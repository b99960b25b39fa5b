"""Refcounted slots of recurrent state, beside the KV pages.

A model with recurrent layers keeps, per sequence, one slot of the engine's state pool.  A step never changes a slot in
place: it reads the sequence's slot and writes a fresh one, which replaces it when the step is committed.  So a step can
be repeated, the rows of a rejected draft are undone by keeping the old slot, and a slot can be shared: a prefix-cache
snapshot holds a reference, and a sequence that resumes from it simply starts reading there.  Slot 0 is the zero state
(never written), slot 1 takes the writes of dummy steps.
"""
from __future__ import annotations

from .paged import Sequence

ZERO_SLOT, SCRATCH_SLOT, FIRST_SLOT = 0, 1, 2


class OutOfSlots(RuntimeError):
    pass


class StatePool:
    def __init__(self, num_slots: int):
        assert num_slots > FIRST_SLOT
        self.num_slots = num_slots
        self.refs = [1 << 30] * FIRST_SLOT + [0] * (num_slots - FIRST_SLOT)
        self.free = list(range(num_slots - 1, FIRST_SLOT - 1, -1))
        self.on_exhausted = None                 # callable() -> bool: give a slot back (evict a snapshot)

    @property
    def free_slots(self) -> int:
        return len(self.free)

    def alloc(self) -> int:
        while not self.free and self.on_exhausted is not None and self.on_exhausted():
            pass
        if not self.free:
            raise OutOfSlots("recurrent state slots exhausted")
        s = self.free.pop()
        self.refs[s] = 1
        return s

    def retain(self, s: int) -> None:
        if s >= FIRST_SLOT:
            assert self.refs[s] > 0, s
            self.refs[s] += 1

    def release(self, s: int) -> None:
        if s >= FIRST_SLOT:
            assert self.refs[s] > 0, s
            self.refs[s] -= 1
            if self.refs[s] == 0:
                self.free.append(s)

    # ---- a step over several sequences ------------------------------------------------------------------------------
    def begin(self, seqs: list[Sequence]) -> tuple[list[int], list[int]]:
        """(slots read, slots written) of one step.  Nothing changes on the sequences yet."""
        outs: list[int] = []
        try:
            for _ in seqs:
                outs.append(self.alloc())
        except OutOfSlots:
            self.abort(outs)
            raise
        return [s.state for s in seqs], outs

    def abort(self, outs: list[int]) -> None:
        for o in outs:
            self.release(o)

    def commit(self, seqs: list[Sequence], outs: list[int], keep_old: bool = False) -> None:
        """The step's slots become the sequences' states.  ``keep_old``: the old slot stays until ``settle`` says how
        many of the step's tokens count."""
        for s, o in zip(seqs, outs):
            self.drop_old(s)
            if keep_old:
                s.old_state = (s.state, s.state_len)
            else:
                self.release(s.state)
            s.state, s.state_len = o, s.kv_len

    def drop_old(self, s: Sequence) -> None:
        if s.old_state is not None:
            self.release(s.old_state[0])
            s.old_state = None

    def settle(self, s: Sequence, length: int) -> None:
        """``length`` tokens of the sequence count.  When the newest slot has seen more, the old one is taken back; the
        tokens between it and ``length`` are run again by the next step (``Sequence.lag``)."""
        if length < s.state_len:
            if s.old_state is None or s.old_state[1] > length:
                raise ValueError(f"recurrent state at {s.state_len} tokens cannot return to {length}")
            self.release(s.state)
            s.state, s.state_len = s.old_state
            s.old_state = None
        else:
            self.drop_old(s)

    def close(self, s: Sequence) -> None:
        self.drop_old(s)
        self.release(s.state)
        s.state, s.state_len = ZERO_SLOT, 0
