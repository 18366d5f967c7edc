"""Plain, slow implementation of the Sumevik decoder: whole sequences, no cache, no batching, one function per mechanism,
float64 on the CPU.  It shares no code with the package under test: its own config.json reading, its own safetensors
reading and its own arithmetic.  In this file's notation (rms_e(x) = sqrt(mean(x^2) + e), sg = logistic function,
ge(z) = z / 2 (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))), positions i, j count from 0):

    stream    : x = E[token];  x <- x + mixer(n1(x));  x <- x + ff(n2(x)) (if the layer has one);  n(x) = x / rms(x) (1 + w)
    gated lru : y = ge(Wy h + by);  p = Wx h + bx;  u_t = sum_m c[:, m] p_(t - K + 1 + m) + cb (p = 0 before the start);
                per part b of `blocks`:  r = sg(Ra_b u_b + ra_b),  i = sg(Ri_b u_b + ri_b);  l = -8 r ln(1 + e^lam);
                S_t = e^l S_(t-1) + sqrt(1 - e^(2 l)) i u;  out = Wo (S * y)
    left      : q, k, v = W. h + b.;  q, k <- x / rms(x) w per head, then turned: pairs (2m, 2m + 1), m < dims / 2, by the
                angle i base^(-2m / dims);  j <= i in i's chunk of C positions;  softmax(scale q_i . k_j);
                Wo (concat_h(o_h) * sg(Wg h))
    right     : q = Wq h / sqrt(dim), k = Wk h, v = Wv h;  d = sg(Wa2 Wa1 h + ab)^(1 / tau);  S_t = diag(d) S_(t-1) + k v^T;
                o = S^T q per head;  Wo (concat_h(o_h / rms(o_h) w) * silu(Wg h))
    parallel  : left_scale * left(h) + right_scale * right(h)
    dense     : Wd (ge(Wg h) * (Wu h))
    experts   : s = softmax(Wr h) over E experts and the identity outputs behind them;  choice score c = s + correction;
                only experts of the `keep` groups with the largest best c;  the `top` largest c;
                weights s / (sum of the chosen s + 1e-20);  an expert is Wd (g sg(1.702 g) (u + 1)), g = min(Wg h, L),
                u = clamp(Wu h, -L, L);  an identity expert is h
    logits    = E n(x) * logit_scale

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

def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(p, taps, bias):
    """p [T, C], taps [C, K] with the last column on the current token; zeros before the start."""
    T, C = p.shape
    K = taps.shape[1]
    out = torch.zeros_like(p) + bias
    for m in range(K):
        back = K - 1 - m
        if back < T:
            out[back:] += taps[:, m] * p[:T - back]
    return out


def lru_gates(u, w, p):
    """(r, i) of every token and channel: each part of the channels has its own two square matrices."""
    ra, ri = w[p + "ra"], w[p + "ri"]
    parts = u.view(u.shape[0], ra.shape[0], ra.shape[1])
    r = torch.sigmoid(torch.einsum("tbc,boc->tbo", parts, ra) + w[p + "ra.b"])
    i = torch.sigmoid(torch.einsum("tbc,boc->tbo", parts, ri) + w[p + "ri.b"])
    return r.reshape(u.shape), i.reshape(u.shape)


def lru_log_decay(r, lam):
    return -8.0 * r * torch.log1p(torch.exp(lam))


def lru_scan(log_a, inp):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) inp_t."""
    S, out = torch.zeros_like(inp[0]), torch.zeros_like(inp)
    a = torch.exp(log_a)
    for t in range(inp.shape[0]):
        S = a[t] * S + torch.sqrt(1.0 - a[t] * a[t]) * inp[t]
        out[t] = S
    return out


def gated_lru(h, w, p, m, rnd=identity):
    y = rnd(gelu_tanh(rnd(h @ w[p + "y"].T) + w[p + "y.b"]))
    x = rnd(h @ w[p + "x"].T) + w[p + "x.b"]
    u = rnd(causal_conv(x, w[p + "conv"], w[p + "conv.b"]))
    r, i = lru_gates(u, w, p)
    S = lru_scan(lru_log_decay(r, w[p + "lam"]), i * u)
    return rnd(rnd(S * y) @ w[p + "o"].T)


def turn_pairs(x, positions, dims, base):
    """x [T, ..., d]: the first `dims` elements turn in pairs (2m, 2m + 1) by the angle position * base^(-2m / dims)."""
    if not dims:
        return x
    m = torch.arange(dims // 2, dtype=F)
    angle = positions.to(F)[:, None] * base ** (-2.0 * m / dims)
    while angle.dim() < x.dim():
        angle = angle.unsqueeze(1)
    c, s = angle.cos(), angle.sin()
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def chunk_visible(T, size):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def chunked_attention(h, w, p, m, eps, rnd=identity):
    """The gated heads side by side, before the output projection."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (rnd(h @ w[p + "q"].T) + w[p + "q.b"]).view(T, H, dk)
    k = (rnd(h @ w[p + "k"].T) + w[p + "k.b"]).view(T, G, dk)
    v = rnd(rnd(h @ w[p + "v"].T) + w[p + "v.b"]).view(T, G, dv)
    rot = m.get("rot") or {}
    q = rnd(turn_pairs(unit_rms(q, eps) * w[p + "q.norm"], pos, rot.get("dims", 0), rot.get("base", 1.0)))
    k = rnd(turn_pairs(unit_rms(k, eps) * w[p + "k.norm"], pos, rot.get("dims", 0), rot.get("base", 1.0)))
    vis = chunk_visible(T, m["mask"]["size"])
    out = torch.zeros(T, H, dv, dtype=F)
    for hh in range(H):
        g = hh // (H // G)
        s = ((q[:, hh] @ k[:, g].T) * m["scale"]).masked_fill(~vis, -math.inf)
        out[:, hh] = torch.softmax(s, dim=1) @ v[:, g]
    return out.reshape(T, H * dv) * torch.sigmoid(rnd(h @ w[p + "g"].T))


def channel_decay(z, tau):
    return torch.sigmoid(z) ** (1.0 / tau)


def linear_scan(q, k, v, decay):
    """q, k, decay [T, H, dk], v [T, H, dv]: S_t = diag(decay_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out


def gated_linear_attention(h, w, p, m, eps, rnd=identity):
    """The normed and gated heads side by side, before the output projection."""
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = rnd(h @ w[p + "q"].T).view(T, H, dk) * dk ** -0.5
    k = rnd(h @ w[p + "k"].T).view(T, H, dk)
    v = rnd(h @ w[p + "v"].T).view(T, H, dv)
    z = rnd(h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    o = linear_scan(q, k, v, channel_decay(z, m["tau"]).view(T, H, dk))
    g = rnd(h @ w[p + "g"].T)
    return (unit_rms(o, eps) * w[p + "norm"]).reshape(T, H * dv) * (g * torch.sigmoid(g))


def side_by_side(h, w, p, m, eps, rnd=identity):
    left = rnd(m["left_scale"] * chunked_attention(h, w, p + "left.", m["left"], eps, rnd)) @ w[p + "left.o"].T
    right = rnd(m["right_scale"] * gated_linear_attention(h, w, p + "right.", m["right"], eps, rnd)) @ w[p + "right.o"].T
    return rnd(left + right)


def dense(h, w, p, rnd=identity):
    a = rnd(gelu_tanh(rnd(h @ w[p + "gate"].T)) * rnd(h @ w[p + "up"].T))
    return rnd(a @ w[p + "down"].T)


def expert(h, w, p, limit, rnd=identity):
    g = torch.clamp(rnd(h @ w[p + "gate"].T), max=limit)
    u = torch.clamp(rnd(h @ w[p + "up"].T), min=-limit, max=limit)
    return rnd(rnd(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T)


def choose(s, correction, router):
    """(ids [T, top], margin [T]): the chosen experts, and by how much the closest decision (between groups, or between the last
    chosen and the first left out) was taken."""
    c = s + correction
    T, N = c.shape
    groups = router.get("groups") or {"count": 1, "keep": 1}
    count, keep = groups["count"], groups["keep"]
    best = c.view(T, count, N // count).max(dim=2).values
    order = torch.argsort(best, dim=1, descending=True)
    margin = torch.full((T,), math.inf, dtype=F)
    if keep < count:
        ranked = best.gather(1, order)
        margin = ranked[:, keep - 1] - ranked[:, keep]
    allowed = torch.zeros(T, count, dtype=torch.bool)
    allowed.scatter_(1, order[:, :keep], True)
    c = c.masked_fill(~allowed.repeat_interleave(N // count, dim=1), -math.inf)
    ranked, ids = torch.sort(c, dim=1, descending=True)
    top = router["top"]
    if top < N:
        margin = torch.minimum(margin, ranked[:, top - 1] - ranked[:, top])
    return ids[:, :top], margin


def routed_experts(h, w, p, f, rnd=identity, margins=None):
    """`margins` (a list) receives, per token, how clear the closest decision of the router was."""
    router = f["router"]
    E, top = router["experts"], router["top"]
    s = torch.softmax(h @ w[p + "router"].T, dim=1)
    ids, margin = choose(s, w[p + "correction"], router)
    if margins is not None:
        margins.append(margin)
    picked = s.gather(1, ids)
    weights = picked / (picked.sum(dim=1, keepdim=True) + 1e-20)
    y = torch.zeros_like(h)
    for c in range(top):
        for e in range(s.shape[1]):
            rows = (ids[:, c] == e).nonzero().flatten()
            if len(rows):
                out = expert(h[rows], w, f"{p}e{e}.", f["expert"]["limit"], rnd) if e < E else h[rows]
                y[rows] += weights[rows, c:c + 1] * out
    return rnd(y)


def forward(model_dir: str, tokens, rnd=identity, return_layers: bool = False):
    """Logits [T, vocab] of one whole sequence (float64); with `return_layers` also the stream after every layer."""
    return forward_loaded(read_config(model_dir), read_weights(model_dir), tokens, rnd, return_layers)


def forward_loaded(cfg, w, tokens, rnd=identity, return_layers: bool = False, router_margins=None):
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    seen = []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rnd(unit_rms(x, eps) * (1.0 + w[p + "norm1"]))
        if layer["type"] == "rglru":
            x = x + gated_lru(h, w, p + "mix.", m, rnd)
        elif layer["type"] == "parallel":
            x = x + side_by_side(h, w, p + "mix.", m, eps, rnd)
        else:
            raise ValueError(f"layer {i}: mixer '{layer['type']}'")
        f = layer.get("mlp")
        if f is not None:
            h = rnd(unit_rms(x, eps) * (1.0 + w[p + "norm2"]))
            x = x + (dense(h, w, p + "mlp.", rnd) if f["kind"] == "dense"
                     else routed_experts(h, w, p + "mlp.", f, rnd, router_margins))
        seen.append(x)
    logits = (rnd(unit_rms(x, eps) * (1.0 + w["final.norm"]) * cfg["logit_scale"])) @ w["embed"].T
    return (logits, torch.stack(seen)) if return_layers else logits
