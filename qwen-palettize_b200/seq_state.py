"""Per-sequence state of a decoder: cached keys and values, recurrent states, convolution inputs. A SequenceState belongs to B sequences
that advance in lockstep; a StatePool hands states to requests and takes them back when they end, so that a served stream of requests
reuses a few allocations."""
from __future__ import annotations

import torch


class SequenceState:
    def __init__(self, specs, B: int, T_max: int, dtype: torch.dtype, device):
        """specs: per layer a dict name -> mixers.StateSpec."""
        self.B, self.capacity, self.length = B, T_max, 0
        self.pos = torch.zeros(1, dtype=torch.int32, device=device)       # the length, for kernels
        self.layers, self._zero = [], []
        for spec in specs:
            st = {}
            for name, s in spec.items():
                shape = tuple(T_max if d == "T_max" else d for d in s.shape)
                st[name] = torch.zeros((B,) + shape, dtype=torch.float32 if s.fp32 else dtype, device=device)
                if s.zero:
                    self._zero.append(st[name])
            self.layers.append(st)
        self.step_graph = None      # captured one-token step over these tensors (hybrid_model)

    def reset(self):
        """Start over: what must begin at zero is cleared; cached keys and values beyond the length are never read."""
        self.length = 0
        self.pos.zero_()
        for t in self._zero:
            t.zero_()

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for st in self.layers for t in st.values())


class StatePool:
    """States of one sequence each, for requests that come and go."""

    def __init__(self, model, capacity: int):
        self.model, self.capacity = model, capacity
        self.free, self.live = [], {}

    def acquire(self, rid):
        if rid in self.live:
            raise ValueError(f"request {rid!r} holds a state already")
        st = self.free.pop() if self.free else self.model.new_cache(1, self.capacity)
        st.reset()
        self.live[rid] = st
        return st

    def get(self, rid):
        return self.live[rid]

    def __contains__(self, rid) -> bool:
        return rid in self.live

    def release(self, rid):
        self.free.append(self.live.pop(rid))

    def tokens_live(self) -> int:
        return sum(s.length for s in self.live.values())
