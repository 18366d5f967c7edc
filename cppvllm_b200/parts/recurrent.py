"""Mixers that carry a matrix per request and head from token to token (fixed-size state in the request's state slot, float32,
zero at admission) instead of a cache that grows with the sequence.  The recurrences run in float32 whatever the activations'
type; only the projections around them are products in the activations' type.

* ``lightning``: q = silu(Wq x), k = silu(Wk x), v = silu(Wv x), heads side by side;  S <- decay_h S + k v^T;  o = S^T q;
  y = Wo (RMSNorm(concat_h o) * w * sigmoid(Wg x)).  State per request: [H, dim, vdim].
* ``channel_delta``: q = Wq x, k = Wk x (kv_heads x dim), v = Wv x (heads x vdim), each through a short causal convolution
  over time per channel (weights [channels, taps], last tap on the current token) and silu; q and k unit vectors per head
  (x / sqrt(sum x^2 + 1e-6)), q also times dim^-1/2; b = sigmoid(Wb x) per head; g = exp(-exp(A_h) * softplus(Wa2 Wa1 x + dt))
  per head and key channel;  S <- diag(g) S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q (head h reads q/k head
  h / (heads / kv_heads));  y = Wo concat_h(RMSNorm(o_h) * w * sigmoid(Wg2 Wg1 x)_h), w shared by the heads.  State per request:
  [H, dim, vdim] and behind it the last taps - 1 inputs of the convolutions [taps - 1, channels].  The inner sizes of the
  two low-rank projections are whatever the checkpoint holds.
* ``head_delta``: the same rule with ONE decay per head and token, g = exp(-exp(A_h) * softplus(Wa x + dt_h)), S <- g S, full-rank
  projections for the decay (Wa [H, D]) and the output gate (Wg [H * vdim, D]), and the gate through silu instead of the
  logistic function: y = Wo concat_h(RMSNorm(o_h) * w * silu(Wg x)_h).
* ``gated_linear``: q = Wq x * dim^-1/2, k = Wk x, v = Wv x; g = sigmoid(Wa2 Wa1 x + b)^(1 / tau) per head and key channel;
  S <- diag(g) S + k v^T;  o = S^T q;  y = Wo concat_h(RMSNorm(o_h) * w * silu(Wg x)_h), w shared by the heads.  State per request:
  [H, dim, vdim].  A step of decoded tokens is one kernel between the projections.  The inner size of the low-rank projection is
  whatever the checkpoint holds.
* ``ssd``: [z | u | dt] = Win x;  [x | B | C] = silu(causal convolution of u over time per channel + bias);  dt <- softplus(dt + dt_bias) per head;
  S <- exp(-exp(A_h) dt) S + dt B x^T  ([state, vdim], B and C of group h / (heads / groups));  y = S^T C + D_h x;
  out = Wo (RMSNorm_parts(y * silu(z)) * w), the norm over ``norm_parts`` equal parts of the row, the gate in front of it.  State per
  request: S of every head and behind it a ring of the last ``taps`` inputs of the convolution.  Portions in bf16 run in chunks on the tensor
  cores, decoded tokens in one kernel and the norm; float32 and other sizes take the token-by-token scan (csrc/ssd.cu, csrc/recurrent.cu).
"""
from __future__ import annotations

from typing import Dict, Optional, Sequence

import torch

from ..csrc import ops
from .base import Mixer, StateSpec, WeightSpec, register_part


def _project(rt, x, w, out, rows):
    return ops.linear(x, w, out=out) if rt.plain_kernels else ops.project_rows(x, w, out, rows)


def _cat_rows(rows):
    if len({r.dtype for r in rows}) > 1:
        rows = [r.float() for r in rows]
    return torch.cat(rows, dim=0).contiguous()


@register_part("mixer", "lightning")
class LightningMixer(Mixer):
    def __init__(self, runtime, prefix="", names=None, *, hidden_size: int, num_heads: int, dim: int, vdim: int,
                 decay: Sequence[float], eps: float):
        super().__init__(runtime, prefix, names)
        self.hidden_size, self.num_heads, self.dim, self.vdim, self.eps = int(hidden_size), int(num_heads), int(dim), int(vdim), float(eps)
        if len(decay) != self.num_heads:
            raise ValueError(f"{len(decay)} decays for {self.num_heads} heads")
        if self.dim > 256:
            raise ValueError("the scan kernel keeps at most 256 key channels per head")
        self.decay = torch.tensor([float(d) for d in decay], dtype=torch.float32, device=runtime.device)
        self.w_in = self.w_o = self.w_norm = None

    def state_spec(self) -> StateSpec:
        return StateSpec((self.num_heads * self.dim * self.vdim,), torch.float32)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        D, H, dk, dv = self.hidden_size, self.num_heads, self.dim, self.vdim
        return {self.full_name("q"): WeightSpec((H * dk, D)), self.full_name("k"): WeightSpec((H * dk, D)),
                self.full_name("v"): WeightSpec((H * dv, D)), self.full_name("g"): WeightSpec((H * dv, D)),
                self.full_name("o"): WeightSpec((D, H * dv)),
                self.full_name("norm"): WeightSpec((H * dv,), role="vector", init="norm")}

    def bind(self, tensors) -> None:
        t = lambda n: tensors[self.full_name(n)]          # noqa: E731
        self.w_in = _cat_rows([t("q"), t("k"), t("v"), t("g")])
        self.w_o, self.w_norm = t("o"), t("norm")

    def weight_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_o))

    def forward(self, x, ctx, cache, state):
        T = x.shape[0]
        H, dk, dv = self.num_heads, self.dim, self.vdim
        ws = self.rt.workspace
        packed = _project(self.rt, x, self.w_in, ws.rows("rec_in", T, self.w_in.shape[0], x.dtype), T)
        f32 = torch.float32
        qf, kf, vf = ws.rows("delta_q", T, H * dk, f32), ws.rows("delta_k", T, H * dk, f32), ws.rows("delta_v", T, H * dv, f32)
        ops.lightning_prep(qf, kf, vf, packed, 0, H * dk, 2 * H * dk)
        o = ws.rows("rec_o", T, H * dv, f32)
        ops.lightning_scan(o, qf, kf, vf, state, self.decay, ctx.cu_seqlens, ctx.state_slots, ctx.num_seqs, H, dk, dv)
        g_off = 2 * H * dk + H * dv
        y = ops.gated_norm(ws.rows("rec_y", T, H * dv, x.dtype), o, packed[:, g_off:g_off + H * dv], self.w_norm, 1, self.eps)
        return _project(self.rt, y, self.w_o, ws.rows("attn_proj", T, self.hidden_size, x.dtype), T)


@register_part("mixer", "channel_delta")
class ChannelDeltaMixer(Mixer):
    def __init__(self, runtime, prefix="", names=None, *, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int,
                 taps: int, eps: float, decay_rank: Optional[int] = None, gate_rank: Optional[int] = None):
        super().__init__(runtime, prefix, names)
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.dim, self.vdim, self.taps, self.eps = int(dim), int(vdim), int(taps), float(eps)
        if self.num_heads % self.num_kv_heads:
            raise ValueError(f"{self.num_heads} heads are not a multiple of {self.num_kv_heads} query/key heads")
        if self.taps < 1:
            raise ValueError("a convolution has at least one tap")
        if self.dim > 256:
            raise ValueError("the scan kernel keeps at most 256 key channels per head")
        self.decay_rank = int(decay_rank) if decay_rank else -1
        self.gate_rank = int(gate_rank) if gate_rank else -1
        self.channels = 2 * self.num_kv_heads * self.dim + self.num_heads * self.vdim
        self.matrix_floats = self.num_heads * self.dim * self.vdim

    def state_spec(self) -> StateSpec:
        return StateSpec((self.matrix_floats + (self.taps - 1) * self.channels,), torch.float32)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        D, H, G, dk, dv, K = self.hidden_size, self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.taps
        f = self.full_name
        return {f("q"): WeightSpec((G * dk, D)), f("q.conv"): WeightSpec((G * dk, K), role="vector"),
                f("k"): WeightSpec((G * dk, D)), f("k.conv"): WeightSpec((G * dk, K), role="vector"),
                f("v"): WeightSpec((H * dv, D)), f("v.conv"): WeightSpec((H * dv, K), role="vector"),
                f("b"): WeightSpec((H, D)), f("A_log"): WeightSpec((H,), role="vector"),
                f("norm"): WeightSpec((dv,), role="vector", init="norm"),
                f("a1"): WeightSpec((self.decay_rank, D)), f("a2"): WeightSpec((H * dk, self.decay_rank)),
                f("dt_bias"): WeightSpec((H * dk,), role="vector"),
                f("g1"): WeightSpec((self.gate_rank, D)), f("g2"): WeightSpec((H * dv, self.gate_rank)),
                f("o"): WeightSpec((D, H * dv))}

    def bind(self, tensors) -> None:
        t = lambda n: tensors[self.full_name(n)]          # noqa: E731
        self.decay_rank, self.gate_rank = t("a1").shape[0], t("g1").shape[0]
        if t("a2").shape[1] != self.decay_rank or t("g2").shape[1] != self.gate_rank:
            raise ValueError(f"{self.prefix}: the two halves of a low-rank projection disagree about its inner size")
        self.w_in = _cat_rows([t("q"), t("k"), t("v"), t("g1"), t("a1")])
        self.g_off = self.channels
        self.a_off = self.channels + self.gate_rank
        self.w_b, self.w_a2, self.w_g2, self.w_o = t("b"), t("a2"), t("g2"), t("o")
        self.conv_w = torch.cat([t("q.conv"), t("k.conv"), t("v.conv")], dim=0).contiguous()
        self.dt_bias, self.a_log, self.w_norm = t("dt_bias"), t("A_log"), t("norm")

    def weight_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_b, self.w_a2, self.w_g2, self.w_o))

    def forward(self, x, ctx, cache, state):
        T, S = x.shape[0], ctx.num_seqs
        H, G, dk, dv = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        ws = self.rt.workspace
        f32 = torch.float32
        packed = _project(self.rt, x, self.w_in, ws.rows("rec_in", T, self.w_in.shape[0], x.dtype), T)
        # what enters the recurrence leaves its product unrounded
        b = ops.linear(x, self.w_b, out=ws.rows("delta_b", T, H, f32), out_dtype=f32)
        a = ops.linear(packed[:, self.a_off:self.a_off + self.decay_rank], self.w_a2, out=ws.rows("delta_a", T, H * dk, f32), out_dtype=f32)
        gate = ops.linear(packed[:, self.g_off:self.g_off + self.gate_rank], self.w_g2, out=ws.rows("delta_gate", T, H * dv, x.dtype))
        qn, kn = ws.rows("delta_q", T, G * dk, f32), ws.rows("delta_k", T, G * dk, f32)
        vv, gg, bb = ws.rows("delta_v", T, H * dv, f32), ws.rows("delta_g", T, H * dk, f32), ws.rows("delta_beta", T, H, f32)
        ops.delta_prep(qn, kn, vv, gg, bb, packed, 0, self.conv_w, a, self.dt_bias, self.a_log, b, state, self.matrix_floats,
                       ctx.seq_of_token, ctx.cu_seqlens, ctx.state_slots, H, G, dk, dv)
        ops.conv_history(state, self.matrix_floats, packed, 0, self.channels, self.taps, ctx.cu_seqlens, ctx.state_slots, S)
        o = ws.rows("rec_o", T, H * dv, f32)
        ops.delta_scan(o, qn, kn, vv, gg, bb, state, ctx.cu_seqlens, ctx.state_slots, S, H, G, dk, dv)
        y = ops.gated_norm(ws.rows("rec_y", T, H * dv, x.dtype), o, gate, self.w_norm, H, self.eps)
        return _project(self.rt, y, self.w_o, ws.rows("attn_proj", T, self.hidden_size, x.dtype), T)


@register_part("mixer", "head_delta")
class HeadDeltaMixer(Mixer):
    def __init__(self, runtime, prefix="", names=None, *, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int,
                 taps: int, eps: float):
        super().__init__(runtime, prefix, names)
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.dim, self.vdim, self.taps, self.eps = int(dim), int(vdim), int(taps), float(eps)
        if self.num_heads % self.num_kv_heads:
            raise ValueError(f"{self.num_heads} heads are not a multiple of {self.num_kv_heads} query/key heads")
        if self.taps < 1:
            raise ValueError("a convolution has at least one tap")
        if self.dim > 256:
            raise ValueError("the scan kernel keeps at most 256 key channels per head")
        self.channels = 2 * self.num_kv_heads * self.dim + self.num_heads * self.vdim
        self.matrix_floats = self.num_heads * self.dim * self.vdim

    def state_spec(self) -> StateSpec:
        return StateSpec((self.matrix_floats + (self.taps - 1) * self.channels,), torch.float32)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        D, H, G, dk, dv, K = self.hidden_size, self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.taps
        f = self.full_name
        return {f("q"): WeightSpec((G * dk, D)), f("q.conv"): WeightSpec((G * dk, K), role="vector"),
                f("k"): WeightSpec((G * dk, D)), f("k.conv"): WeightSpec((G * dk, K), role="vector"),
                f("v"): WeightSpec((H * dv, D)), f("v.conv"): WeightSpec((H * dv, K), role="vector"),
                f("b"): WeightSpec((H, D)), f("a"): WeightSpec((H, D)), f("A_log"): WeightSpec((H,), role="vector"),
                f("dt_bias"): WeightSpec((H,), role="vector"), f("norm"): WeightSpec((dv,), role="vector", init="norm"),
                f("g"): WeightSpec((H * dv, D)), f("o"): WeightSpec((D, H * dv))}

    def bind(self, tensors) -> None:
        t = lambda n: tensors[self.full_name(n)]          # noqa: E731
        self.w_in = _cat_rows([t("q"), t("k"), t("v"), t("g")])
        self.g_off = self.channels
        self.w_b, self.w_a, self.w_o = t("b"), t("a"), t("o")
        self.conv_w = torch.cat([t("q.conv"), t("k.conv"), t("v.conv")], dim=0).contiguous()
        self.dt_bias, self.a_log, self.w_norm = t("dt_bias"), t("A_log"), t("norm")

    def weight_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_b, self.w_a, self.w_o))

    def forward(self, x, ctx, cache, state):
        T, S = x.shape[0], ctx.num_seqs
        H, G, dk, dv = self.num_heads, self.num_kv_heads, self.dim, self.vdim
        ws = self.rt.workspace
        f32 = torch.float32
        packed = _project(self.rt, x, self.w_in, ws.rows("rec_in", T, self.w_in.shape[0], x.dtype), T)
        # what enters the recurrence leaves its product unrounded
        b = ops.linear(x, self.w_b, out=ws.rows("delta_b", T, H, f32), out_dtype=f32)
        a = ops.linear(x, self.w_a, out=ws.rows("delta_a1", T, H, f32), out_dtype=f32)
        qn, kn = ws.rows("delta_q", T, G * dk, f32), ws.rows("delta_k", T, G * dk, f32)
        vv, gg, bb = ws.rows("delta_v", T, H * dv, f32), ws.rows("delta_g1", T, H, f32), ws.rows("delta_beta", T, H, f32)
        ops.delta_prep(qn, kn, vv, gg, bb, packed, 0, self.conv_w, a, self.dt_bias, self.a_log, b, state, self.matrix_floats,
                       ctx.seq_of_token, ctx.cu_seqlens, ctx.state_slots, H, G, dk, dv, decay_dim=1)
        ops.conv_history(state, self.matrix_floats, packed, 0, self.channels, self.taps, ctx.cu_seqlens, ctx.state_slots, S)
        o = ws.rows("rec_o", T, H * dv, f32)
        ops.delta_scan(o, qn, kn, vv, gg, bb, state, ctx.cu_seqlens, ctx.state_slots, S, H, G, dk, dv, decay_dim=1)
        y = ops.gated_norm(ws.rows("rec_y", T, H * dv, x.dtype), o, packed[:, self.g_off:self.g_off + H * dv], self.w_norm, H, self.eps,
                           gate_act="silu")
        return _project(self.rt, y, self.w_o, ws.rows("attn_proj", T, self.hidden_size, x.dtype), T)


@register_part("mixer", "gated_linear")
class GatedLinearMixer(Mixer):
    def __init__(self, runtime, prefix="", names=None, *, hidden_size: int, num_heads: int, dim: int, vdim: int, tau: float, eps: float,
                 decay_rank: Optional[int] = None):
        super().__init__(runtime, prefix, names)
        self.hidden_size, self.num_heads, self.dim, self.vdim = int(hidden_size), int(num_heads), int(dim), int(vdim)
        self.tau, self.eps = float(tau), float(eps)
        self.decay_rank = int(decay_rank) if decay_rank else -1
        if self.dim > 512:
            raise ValueError("the scan kernel keeps at most 512 key channels per head")
        self.core_width = self.num_heads * self.vdim
        self.w_in = self.w_o = self.w_a2 = None

    def state_spec(self) -> StateSpec:
        return StateSpec((self.num_heads * self.dim * self.vdim,), torch.float32)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        D, H, dk, dv, R = self.hidden_size, self.num_heads, self.dim, self.vdim, self.decay_rank
        f = self.full_name
        return {f("q"): WeightSpec((H * dk, D)), f("k"): WeightSpec((H * dk, D)), f("v"): WeightSpec((H * dv, D)), f("g"): WeightSpec((H * dv, D)),
                f("a1"): WeightSpec((R, D)), f("a2"): WeightSpec((H * dk, R)), f("a2.b"): WeightSpec((H * dk,), role="vector"),
                f("norm"): WeightSpec((dv,), role="vector", init="norm"), f("o"): WeightSpec((D, H * dv))}

    def bind(self, tensors) -> None:
        t = lambda n: tensors[self.full_name(n)]          # noqa: E731
        self.decay_rank = t("a1").shape[0]
        if t("a2").shape[1] != self.decay_rank:
            raise ValueError(f"{self.prefix}: the two halves of the low-rank projection disagree about its inner size")
        self.w_in = _cat_rows([t("q"), t("k"), t("v"), t("g"), t("a1")])
        self.w_a2, self.b_a2, self.w_norm, self.w_o = t("a2"), t("a2.b").contiguous(), t("norm").contiguous(), t("o")
        self._scaled = (1.0, self.w_norm)

    def inner_weight_bytes(self) -> int:
        return self.w_a2.numel() * self.w_a2.element_size()

    def weight_bytes(self) -> int:
        return self.inner_weight_bytes() + sum(w.numel() * w.element_size() for w in (self.w_in, self.w_o))

    def forward(self, x, ctx, cache, state):
        T = x.shape[0]
        ws = self.rt.workspace
        packed = _project(self.rt, x, self.w_in, ws.rows("rec_in", T, self.w_in.shape[0], x.dtype), T)
        y = self.core(packed, ws.rows("rec_y", T, self.core_width, x.dtype), 1.0, ctx, cache, state)
        return _project(self.rt, y, self.w_o, ws.rows("attn_proj", T, self.hidden_size, x.dtype), T)

    def core(self, packed, out, scale, ctx, cache, state):
        T, S = packed.shape[0], ctx.num_seqs
        H, dk, dv, R = self.num_heads, self.dim, self.vdim, self.decay_rank
        q_off, k_off, v_off, g_off, a_off = 0, H * dk, 2 * H * dk, 2 * H * dk + H * dv, 2 * H * dk + 2 * H * dv
        qk_scale = dk ** -0.5
        if (ctx.all_decode and T == S and not self.rt.plain_kernels and self.w_a2.dtype == packed.dtype
                and ops.linear_step_supported(dk, dv, R)):
            return ops.linear_step(out, packed, q_off, k_off, v_off, g_off, a_off, self.w_a2, self.b_a2, qk_scale, self.tau, self.w_norm,
                                   self.eps, scale, state, ctx.cu_seqlens, ctx.state_slots, S, H, dk, dv)
        ws, f32 = self.rt.workspace, torch.float32
        # the decay's logits leave their product unrounded and become the decays in place
        z = ops.linear(packed[:, a_off:a_off + R], self.w_a2, out=ws.rows("linear_g", T, H * dk, f32), out_dtype=f32)
        ops.linear_decay(z, self.b_a2, self.tau)
        o = ws.rows("rec_o", T, H * dv, f32)
        q_lens = ctx.q_lens if ctx.q_lens is not None else [1] * S
        chunk = ops.linear_chunk_tokens(T, H, dk, dv)
        ends = decays = None
        if max(q_lens) > chunk:
            held = ops.linear_held_chunks(ws.max_tokens, H, dk, dv)
            ends = ws.flat(f"linear_ends_{H}_{dk}_{dv}", held * H * dk * dv, f32)
            decays = ws.flat(f"linear_decays_{H}_{dk}_{dv}", held * H * dk, f32)
        ops.linear_scan(o, packed, q_off, k_off, v_off, qk_scale, z, state, ctx.cu_seqlens, ctx.state_slots, q_lens, H, dk, dv, chunk, ends, decays)
        if self._scaled[0] != scale:                      # the constant rides on the norm's weight
            self._scaled = (scale, (self.w_norm * scale).contiguous())
        return ops.gated_norm(out, o, packed[:, g_off:g_off + H * dv], self._scaled[1], H, self.eps, gate_act="silu")


@register_part("mixer", "ssd")
class StateSpaceMixer(Mixer):
    def __init__(self, runtime, prefix="", names=None, *, hidden_size: int, num_heads: int, groups: int, state: int, vdim: int, taps: int,
                 norm_parts: int, eps: float):
        super().__init__(runtime, prefix, names)
        self.hidden_size, self.num_heads, self.groups, self.dim, self.vdim = int(hidden_size), int(num_heads), int(groups), int(state), int(vdim)
        self.taps, self.norm_parts, self.eps = int(taps), int(norm_parts), float(eps)
        if self.num_heads % self.groups:
            raise ValueError(f"{self.num_heads} heads are not a multiple of {self.groups} groups")
        self.inner = self.num_heads * self.vdim
        if self.inner % self.norm_parts:
            raise ValueError(f"{self.inner} columns do not fall into {self.norm_parts} equal parts")
        if self.taps < 1:
            raise ValueError("a convolution has at least one tap")
        if self.dim > 512:
            raise ValueError("the scan kernel keeps at most 512 rows of a state")
        self.channels = self.inner + 2 * self.groups * self.dim
        self.core_width = self.inner
        self.w_in = self.w_o = None

    def state_spec(self) -> StateSpec:
        n = self.num_heads * self.dim * self.vdim + (self.taps * self.channels if self.taps > 1 else 0)
        return StateSpec((-(-n // 4) * 4,), torch.float32)           # whole 16-byte pieces: every slot's matrices start on one

    def weight_specs(self) -> Dict[str, WeightSpec]:
        D, H, C = self.hidden_size, self.num_heads, self.channels
        f = self.full_name
        return {f("in"): WeightSpec((self.inner + C + H, D)), f("conv"): WeightSpec((C, self.taps), role="vector"), f("conv.b"): WeightSpec((C,), role="vector"),
                f("dt_bias"): WeightSpec((H,), role="vector"), f("A_log"): WeightSpec((H,), role="vector"), f("D"): WeightSpec((H,), role="vector", init="norm"),
                f("norm"): WeightSpec((self.inner,), role="vector", init="norm"), f("o"): WeightSpec((D, self.inner))}

    def bind(self, tensors) -> None:
        t = lambda n: tensors[self.full_name(n)]          # noqa: E731
        self.w_in, self.w_o = t("in"), t("o")
        self.conv_w, self.conv_b = t("conv").t().contiguous(), t("conv.b").contiguous()
        self.dt_bias, self.neg_a, self.skip, self.w_norm = t("dt_bias").contiguous(), (-torch.exp(t("A_log"))).contiguous(), t("D").contiguous(), t("norm").contiguous()

    def weight_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_o))

    def forward(self, x, ctx, cache, state):
        T = x.shape[0]
        ws = self.rt.workspace
        packed = _project(self.rt, x, self.w_in, ws.rows("rec_in", T, self.w_in.shape[0], x.dtype), T)
        y = self.core(packed, ws.rows("rec_y", T, self.core_width, x.dtype), 1.0, ctx, cache, state)
        return _project(self.rt, y, self.w_o, ws.rows("attn_proj", T, self.hidden_size, x.dtype), T)

    def core(self, packed, out, scale, ctx, cache, state):
        T, S = packed.shape[0], ctx.num_seqs
        sizes = (self.num_heads, self.groups, self.dim, self.vdim)
        H, G, N, P = sizes
        ws, f32 = self.rt.workspace, torch.float32
        u_off, dt_off = self.inner, self.inner + self.channels
        y = ws.rows("rec_o", T, self.inner, f32)
        if ctx.all_decode and T == S and not self.rt.plain_kernels and ops.ssd_step_supported(N, P):
            ops.ssd_step(y, packed, u_off, dt_off, self.conv_w, self.conv_b, self.dt_bias, self.neg_a, self.skip, state, ctx.cu_seqlens,
                         ctx.state_slots, ctx.positions, S, *sizes)
        else:
            q_lens = ctx.q_lens if ctx.q_lens is not None else [1] * S
            chunks = not self.rt.plain_kernels and ops.ssd_chunks_supported(packed.dtype, N, P)
            u = ws.rows("ssd_u", T, self.channels, packed.dtype if chunks else f32)
            dt, la = ws.rows("ssd_dt", T, H, f32), ws.rows("ssd_log_decay", T, H, f32)
            ops.ssd_prep(u, dt, la, packed, u_off, dt_off, self.conv_w, self.conv_b, self.dt_bias, self.neg_a, state, ctx.seq_of_token,
                         ctx.cu_seqlens, ctx.state_slots, ctx.positions, *sizes)
            ops.ssd_ring(state, packed, u_off, dt_off, self.taps, ctx.cu_seqlens, ctx.state_slots, ctx.positions, S, *sizes)
            if chunks:
                ends = decays = None
                if max(q_lens) > ops.SSD_CHUNK:
                    held = ops.ssd_held_chunks(ws.max_tokens)
                    ends = ws.flat(f"ssd_ends_{H}_{N}_{P}", held * H * N * P, f32)
                    decays = ws.flat(f"ssd_decays_{H}", held * H, f32)
                ops.ssd_chunks(y, u, dt, la, self.skip, state, ctx.cu_seqlens, ctx.state_slots, q_lens, *sizes, ends=ends, decays=decays)
            else:
                i, n = self.inner, G * N
                ops.skip_scan(y, u[:, i + n:], u[:, i:i + n], u[:, :i], la, dt, self.skip, state, ctx.cu_seqlens, ctx.state_slots, S, H, G, N, P)
        return ops.gate_norm(out, y, packed[:, :self.inner], self.w_norm, self.norm_parts, self.eps, scale)
