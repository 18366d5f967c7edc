"""Mixer ``gated_lru``: a gated linear recurrence with one number of state per channel, behind a short causal convolution.

    y = gelu_tanh(Wy x + by);   p = Wx x + bx;   u = conv(p) + cb           (causal, per channel; zeros before the sequence's start)
    per part b of `blocks` equal parts of the channels:  r = sigmoid(Ra_b u_b + ra_b),  i = sigmoid(Ri_b u_b + ri_b)
    l = -8 r softplus(lam);   S_t = e^l S_(t-1) + sqrt(1 - e^(2 l)) i u;    out = Wo (S * y)

The recurrence and its gates run in float32 whatever the activations' type; u is rounded once to the activations' type, as the
operand of the gate products.  State per request: S [W] and, with more than one tap, a ring of the last `taps` inputs p
[taps, W] by position (csrc/lru.cu).  A step of few decoded tokens is one kernel between the two projections; other steps
run the convolution, one batched product for both gates of every part, and the scan over chunks of tokens side by side.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..csrc import ops
from .base import Mixer, StateSpec, WeightSpec, register_part
from .recurrent import _cat_rows, _project


@register_part("mixer", "gated_lru")
class GatedLRUMixer(Mixer):
    def __init__(self, runtime, prefix="", names=None, *, hidden_size: int, width: int, taps: int, blocks: int, decay_scale: float = 8.0):
        super().__init__(runtime, prefix, names)
        self.hidden_size, self.width, self.taps, self.blocks = int(hidden_size), int(width), int(taps), int(blocks)
        self.decay_scale = float(decay_scale)
        if self.taps < 1:
            raise ValueError("a convolution has at least one tap")
        if self.width % self.blocks:
            raise ValueError(f"{self.width} channels do not split into {self.blocks} equal parts")
        self.w_in = self.w_o = self.gates = None

    def state_spec(self) -> StateSpec:
        return StateSpec((self.width * (1 + (self.taps if self.taps > 1 else 0)),), torch.float32)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        D, W, B = self.hidden_size, self.width, self.blocks
        part = W // B
        f = self.full_name
        return {f("y"): WeightSpec((W, D)), f("y.b"): WeightSpec((W,), role="vector"),
                f("x"): WeightSpec((W, D)), f("x.b"): WeightSpec((W,), role="vector"),
                f("conv"): WeightSpec((W, self.taps), role="vector"), f("conv.b"): WeightSpec((W,), role="vector"),
                f("ra"): WeightSpec((B, part, part)), f("ra.b"): WeightSpec((B, part), role="vector"),
                f("ri"): WeightSpec((B, part, part)), f("ri.b"): WeightSpec((B, part), role="vector"),
                f("lam"): WeightSpec((W,), role="vector"), f("o"): WeightSpec((D, W))}

    def bind(self, tensors) -> None:
        t = lambda n: tensors[self.full_name(n)]          # noqa: E731
        self.w_in, self.w_o = _cat_rows([t("y"), t("x")]), t("o")
        self.b_y, self.b_x = t("y.b").contiguous(), t("x.b").contiguous()
        self.conv_w, self.conv_b = t("conv").float().t().contiguous(), t("conv.b").contiguous()      # by tap, oldest first
        self.gates = torch.cat([t("ra"), t("ri")], dim=1).to(self.rt.dtype).contiguous()             # [blocks, 2 * part, part]
        self.b_r, self.b_i = t("ra.b").reshape(-1).contiguous(), t("ri.b").reshape(-1).contiguous()
        self.neg_softplus = (-self.decay_scale * torch.nn.functional.softplus(t("lam").double())).float().contiguous()

    def weight_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.gates, self.w_o))

    def forward(self, x, ctx, cache, state):
        T, W = x.shape[0], self.width
        ws = self.rt.workspace
        packed = _project(self.rt, x, self.w_in, ws.rows("lru_in", T, 2 * W, x.dtype), T)
        out = ws.rows("lru_out", T, W, x.dtype)
        if ctx.all_decode and T == ctx.num_seqs and T <= ops.LRU_STEP_MAX and not self.rt.plain_kernels:
            ops.lru_step(out, packed, 0, W, self.b_y, self.b_x, self.conv_w, self.conv_b, self.gates, self.b_r, self.b_i, self.neg_softplus,
                         state, ctx.cu_seqlens, ctx.state_slots, ctx.positions, ctx.num_seqs)
        else:
            q_lens = ctx.q_lens if ctx.q_lens is not None else [1] * ctx.num_seqs
            u = ops.lru_conv(ws.rows("lru_u", T, W, x.dtype), packed, 0, W, self.blocks, self.b_x, self.conv_w, self.conv_b, state,
                             ctx.seq_of_token, ctx.cu_seqlens, ctx.state_slots, ctx.positions)
            z = ops.lru_gates(ws.rows("lru_z", T, 2 * W, torch.float32), u, self.gates)
            summary = ws.flat(f"lru_summary_{W}", ops.lru_most_chunks(ws.max_tokens, ws.max_seqs, W) * 2 * W, torch.float32)
            ops.lru_scan(out, z, u, packed, 0, W, self.blocks, self.taps, self.b_y, self.b_x, self.b_r, self.b_i, self.neg_softplus, state,
                         ctx.cu_seqlens, ctx.state_slots, ctx.positions, q_lens, ops.lru_chunk_tokens(T, W), summary)
        return _project(self.rt, out, self.w_o, ws.rows("attn_proj", T, self.hidden_size, x.dtype), T)
