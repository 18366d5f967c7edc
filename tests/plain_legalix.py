"""Plain, slow implementation of the Legalix decoder: whole sequences, no cache, no batching, one function per mechanism,
float64 on the CPU.  It shares no code with the package under test: its own config.json reading, its own safetensors
reading and its own arithmetic.  In this file's notation (rms(x) = sqrt(mean(x^2) + eps), sl(z) = z / (1 + e^-z),
ge(z) = z / 2 (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))), positions i, j count from 0):

    embedding : x = x0 = c E[token]
    run order : layers 0 .. stop - 1, with start .. stop - 1 run `times` times in a row, then the rest; in front of every pass
                x <- Win [x ; x0]
    layer     : h = n(x);  x <- x + m (mixer(h) + ff(h))   (no ff: x + m mixer(h));  n(x) = tanh(a x) w + b
    attention : q, k, v = W. h;  q, k turned: elements e and e + dims / 2 by the angle i base^(-2 e / dims);
                s = cap tanh(scale q_i . k_j / cap);  j <= i and (i - j < size or j < keep_first);  softmax;  Wo concat_h
    latent    : cq = Wdq h / rms w;  q = Wuq cq per head [unturned | turned];  [c | r] = Wdkv h;  c <- c / rms(c) w;
                k_h = Wuk_h c, v_h = Wuv_h c;  turned parts: pairs (2e, 2e + 1);  s = scale (qn . k + qr . r_j);  j <= i;
                weights e^s / (sum_j e^s + e^sink_h);  Wo concat_h
    ssd       : [z | u | dt] = Win h;  u <- sl(causal convolution of u + bias) = [x | B | C];  dt <- ln(1 + e^(dt + bias_h));
                S_t = e^(-e^A_h dt) S_(t-1) + dt B_t x_t^T  (N x vdim, B and C of group h / (heads / groups));
                y = S^T C + D_h x;  y <- y sl(z);  norm_groups equal parts, each by its own rms, times w;  Wo
    ff        : Wd (ge(Wg h) * (Wu h))
    logits    : head n(x)

``rnd`` rounds where a 16-bit implementation would (identity by default)."""
import json
import math
import os
import struct

import numpy as np
import torch

F = torch.float64


def identity(x):
    return x


def to_bf16(x):
    return x.to(torch.float32).to(torch.bfloat16).to(F)


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)


def read_weights(model_dir: str) -> dict:
    """Own reader of the container: 8 bytes of header length, a JSON header, raw little-endian data."""
    out = {}
    with open(os.path.join(model_dir, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        raw = data[meta["data_offsets"][0]:meta["data_offsets"][1]]
        if meta["dtype"] == "BF16":
            a = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16
            t = torch.from_numpy(a.view(np.float32).copy()).to(F)
        elif meta["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(raw, dtype="<f4").copy()).to(F)
        elif meta["dtype"] == "I32":
            t = torch.from_numpy(np.frombuffer(raw, dtype="<i4").copy())
        else:
            raise ValueError(f"{name}: element type {meta['dtype']}")
        out[name] = t.reshape(tuple(meta["shape"]))
    return out


# ---- mechanisms ----------------------------------------------------------------------------------------------------------

def dynamic_tanh(x, w, name):
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def turn(x, positions, dims, base, interleaved):
    """x [T, ..., d]: the first `dims` elements turn in pairs (2e, 2e + 1), or (e, e + dims / 2), by position * base^(-2e / dims)."""
    e = torch.arange(dims // 2, dtype=F)
    angle = positions.to(F)[:, None] * base ** (-2.0 * e / dims)
    while angle.dim() < x.dim():
        angle = angle.unsqueeze(1)
    c, s = angle.cos(), angle.sin()
    first, second = (slice(0, dims, 2), slice(1, dims, 2)) if interleaved else (slice(0, dims // 2), slice(dims // 2, dims))
    u, v = x[..., first], x[..., second]
    out = x.clone()
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


def window_visible(T, size, keep_first):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def capped(s, cap):
    return cap * torch.tanh(s / cap)


def windowed_attention(h, w, p, m, rnd=identity):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q = rnd(turn(rnd(h @ w[p + "q"].T).view(T, H, dk), pos, dims, base, False))
    k = rnd(turn(rnd(h @ w[p + "k"].T).view(T, G, dk), pos, dims, base, False))
    v = rnd(h @ w[p + "v"].T).view(T, G, dv)
    vis = window_visible(T, m["mask"]["size"], m["mask"]["keep_first"])
    out = torch.zeros(T, H, dv, dtype=F)
    for hh in range(H):
        g = hh // (H // G)
        s = capped((q[:, hh] @ k[:, g].T) * m["scale"], m["softcap"]).masked_fill(~vis, -math.inf)
        out[:, hh] = torch.softmax(s, dim=1) @ v[:, g]
    return rnd(rnd(out.reshape(T, H * dv)) @ w[p + "o"].T)


def sink_softmax(s, sink):
    """Softmax over the last axis whose denominator also holds e^sink."""
    top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def latent_attention(h, w, p, m, eps, rnd=identity):
    T = h.shape[0]
    H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    cq = rnd(unit_rms(rnd(h @ w[p + "dq"].T), eps) * w[p + "dq.norm"])
    q = rnd(cq @ w[p + "uq"].T).view(T, H, dn + dr)
    qn, qr = q[..., :dn], rnd(turn(q[..., dn:], pos, dims, base, True))
    down = rnd(h @ w[p + "dkv"].T)
    c = rnd(unit_rms(down[:, :R], eps) * w[p + "dkv.norm"])
    kr = rnd(turn(down[:, R:], pos, dims, base, True))
    kn = rnd(c @ w[p + "uk"].T).view(T, H, dn)
    v = rnd(c @ w[p + "uv"].T).view(T, H, dv)
    causal = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = torch.zeros(T, H, dv, dtype=F)
    for hh in range(H):
        s = ((qn[:, hh] @ kn[:, hh].T + qr[:, hh] @ kr.T) * m["scale"]).masked_fill(~causal, -math.inf)
        out[:, hh] = sink_softmax(s, w[p + "sink"][hh]) @ v[:, hh]
    return rnd(rnd(out.reshape(T, H * dv)) @ w[p + "o"].T)


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K] with the last column on the current token; zeros before the start."""
    T = x.shape[0]
    K = taps.shape[1]
    out = torch.zeros_like(x) + bias
    for m in range(K):
        back = K - 1 - m
        if back < T:
            out[back:] += taps[:, m] * x[:T - back]
    return out


def ssd_scan(x, B, C, dt, a_log, D):
    """x [T, H, P], B and C [T, G, N], dt [T, H]: S_t = exp(-exp(a_log) dt) S_(t-1) + dt B x^T, y = S^T C + D x."""
    T, H, P = x.shape
    per = H // B.shape[1]
    S = torch.zeros(H, B.shape[2], P, dtype=F)
    out = torch.zeros_like(x)
    for t in range(T):
        b, c = B[t].repeat_interleave(per, dim=0), C[t].repeat_interleave(per, dim=0)
        decay = torch.exp(-torch.exp(a_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * b[:, :, None] * x[t][:, None, :]
        out[t] = torch.einsum("hnp,hn->hp", S, c) + D[:, None] * x[t]
    return out


def gated_group_norm(y, z, weight, groups, eps):
    """The gate comes before the norm; every one of `groups` equal parts has its own root mean square."""
    y = y * silu(z)
    return unit_rms(y.view(y.shape[0], groups, -1), eps).reshape(y.shape) * weight


def ssd(h, w, p, m, eps, rnd=identity):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, gn = H * P, G * N
    proj = h @ w[p + "in"].T
    z, u, dt = rnd(proj[:, :inner]), rnd(proj[:, inner:2 * inner + 2 * gn]), proj[:, 2 * inner + 2 * gn:]
    u = silu(causal_conv(u, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = u[:, :inner].view(T, H, P), u[:, inner:inner + gn].view(T, G, N), u[:, inner + gn:].view(T, G, N)
    dt = torch.nn.functional.softplus(dt + w[p + "dt_bias"], threshold=60.0)
    y = ssd_scan(x, B, C, dt, w[p + "A_log"], w[p + "D"]).reshape(T, inner)
    return rnd(rnd(gated_group_norm(y, z, w[p + "norm"], m["norm_groups"], eps)) @ w[p + "o"].T)


def dense(h, w, p, rnd=identity):
    a = rnd(gelu_tanh(rnd(h @ w[p + "gate"].T)) * rnd(h @ w[p + "up"].T))
    return rnd(a @ w[p + "down"].T)


def pass_input(x, x0, w, rnd=identity):
    return rnd(torch.cat([x, x0], dim=1)) @ w["loop.in"].T


def run_order(cfg):
    """(layer, begins a pass) for every layer run."""
    loop = cfg.get("loop")
    n = len(cfg["layers"])
    if not loop:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(loop["start"])]
    for _ in range(loop["times"]):
        order += [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(model_dir: str, tokens, rnd=identity, return_layers: bool = False):
    """Logits [T, vocab] of one whole sequence (float64); with `return_layers` also the stream after every layer run."""
    return forward_loaded(read_config(model_dir), read_weights(model_dir), tokens, rnd, return_layers)


def forward_loaded(cfg, w, tokens, rnd=identity, return_layers: bool = False):
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    seen = []
    for i, begins in run_order(cfg):
        if begins:
            x = pass_input(x, x0, w, rnd)
        layer = cfg["layers"][i]
        p, m = f"l{i}.", layer["mixer"]
        h = rnd(dynamic_tanh(x, w, p + "norm1"))
        if layer["type"] == "attention":
            y = windowed_attention(h, w, p + "mix.", m, rnd)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", m, eps, rnd)
        elif layer["type"] == "mamba2":
            y = ssd(h, w, p + "mix.", m, eps, rnd)
        else:
            raise ValueError(f"layer {i}: mixer '{layer['type']}'")
        if layer.get("mlp") is not None:
            y = y + dense(h, w, p + "mlp.", rnd)
        x = x + mult * y
        seen.append(x)
    logits = rnd(dynamic_tanh(x, w, "final.norm")) @ w["head"].T
    return (logits, torch.stack(seen)) if return_layers else logits
