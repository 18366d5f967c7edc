"""Mixer ``side_by_side``: several mixers (or mixers and a feed-forward: a layer whose two sublayers share one norm) that read the same
input, their outputs added up with a constant each:

    y = sum_m scale_m mixer_m(x)

A member keeps its own tensors, cache entries and state, and offers its middle part, ``core(packed, out, scale, ctx, cache,
state)``: from the columns of its input projection (``w_in``) to ``core_width`` columns in front of its output projection
(``w_o``), times `scale`.  The members' input projections are one product (their rows one below the other), the scaled cores lie
side by side in one buffer, and their output projections are one product too (their columns side by side), whose sum over
the inner dimension is the sum over the members: two products for the layer, and no kernel adds anything up.
The cores share nothing, so every one but the first runs on a stream of its own beside it (inside a captured graph: a fork and
a join), and attention and a recurrence fill the SMs together.  At most one member may keep cache entries and at most one
per-request state.
"""
from __future__ import annotations

from typing import Dict, Sequence

import torch

from ..csrc import ops
from .base import Mixer, WeightSpec, register_part
from .recurrent import _cat_rows, _project

ROW_STEP = 8        # every member's rows of the joined input projection are padded to whole 16-byte chunks of bf16 outputs


@register_part("mixer", "side_by_side")
class SideBySideMixer(Mixer):
    def __init__(self, runtime, prefix="", names=None, *, hidden_size: int, members: Sequence[Mixer], scales: Sequence[float]):
        super().__init__(runtime, prefix, names)
        self.hidden_size, self.members, self.scales = int(hidden_size), tuple(members), tuple(float(s) for s in scales)
        if not self.members or len(self.members) != len(self.scales):
            raise ValueError("one scale per mixer")
        for m in self.members:
            if not hasattr(m, "core"):
                raise ValueError(f"{type(m).__name__} does not offer what lies between its projections")
        if sum(m.cache_spec() is not None for m in self.members) > 1 or sum(m.state_spec() is not None for m in self.members) > 1:
            raise ValueError("at most one of the mixers keeps cache entries, and at most one per-request state")
        self.core_width = sum(m.core_width for m in self.members)
        self.w_in = self.w_o = None
        self._streams = None

    @property
    def capturable(self) -> bool:
        return all(m.capturable for m in self.members)

    def _only(self, specs):
        return next((s for s in specs if s is not None), None)

    def cache_spec(self):
        return self._only(m.cache_spec() for m in self.members)

    def state_spec(self):
        return self._only(m.state_spec() for m in self.members)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        specs: Dict[str, WeightSpec] = {}
        for m in self.members:
            specs.update(m.weight_specs())
        return specs

    def bind(self, tensors) -> None:
        self.in_cols = []
        col, rows = 0, []
        for m in self.members:
            m.bind(tensors)
            n = m.w_in.shape[0]
            self.in_cols.append((col, col + n))
            rows.append(m.w_in)
            pad = -n % ROW_STEP
            if pad:
                rows.append(torch.zeros(pad, self.hidden_size, dtype=m.w_in.dtype, device=m.w_in.device))
            col += n + pad
        self.w_in = _cat_rows(rows)
        outs = [m.w_o for m in self.members]
        if len({o.dtype for o in outs}) > 1:
            outs = [o.float() for o in outs]
        self.w_o = torch.cat(outs, dim=1).contiguous()
        for m in self.members:                # the joined matrices are the ones that are read
            m.w_in = m.w_o = None

    def weight_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_o)) + sum(getattr(m, "inner_weight_bytes", int)() for m in self.members)

    def forward(self, x, ctx, cache, state):
        T = x.shape[0]
        ws = self.rt.workspace
        packed = _project(self.rt, x, self.w_in, ws.rows("pair_in", T, self.w_in.shape[0], x.dtype), T)
        joined = ws.rows("pair_out", T, self.core_width, x.dtype)
        main = torch.cuda.current_stream(x.device)
        if self._streams is None:
            self._streams = [torch.cuda.Stream(x.device) for _ in self.members[1:]]
        beside = not self.rt.plain_kernels
        o0 = 0
        for i, (m, scale, (c0, c1)) in enumerate(zip(self.members, self.scales, self.in_cols)):
            args = (packed[:, c0:c1], joined[:, o0:o0 + m.core_width], scale, ctx, cache, state)
            o0 += m.core_width
            if i == 0 or not beside:
                first = (m, args) if beside else None
                if not beside:
                    m.core(*args)
                continue
            side = self._streams[i - 1]
            side.wait_stream(main)
            with torch.cuda.stream(side):
                m.core(*args)
        if beside:
            first[0].core(*first[1])                      # launched last, on the caller's stream
            for side in self._streams:
                main.wait_stream(side)
        y = ws.rows("attn_proj", T, self.hidden_size, x.dtype)
        if self.rt.plain_kernels:
            return ops.linear(joined, self.w_o, out=y)
        return ops.project_rows(joined, self.w_o, y, T, dependent=False)      # behind the join, not beside it
