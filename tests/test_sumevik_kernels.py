"""The kernels that came with Sumevik, each alone against float64 arithmetic written here or in tests/plain_sumevik.py: biases in
the attention projection's epilogue, a gate per element and an output inside wider rows, the linear-attention scan (whole portions,
portions cut anywhere, chunks side by side) and its form for decoded tokens, the gated recurrence over channels likewise, routing
with a correction inside the best groups, clamped and identity experts, and the gated products."""
import pytest
import torch

import plain_sumevik as plain

pytestmark = pytest.mark.gpu

F = torch.float64
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 3e-5, "bfloat16": 2e-2}


def dev():
    return torch.device("cuda:0")


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=dev())


def close(got, want, tol, what=""):
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.isfinite(got).all(), what
    err = float((got - want).abs().max()) / max(1.0, float(want.abs().max()))
    assert err < tol, f"{what}: {err:.2e}"


# ---- chunked attention: biases, gate per element, constant, output inside wider rows ------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,rot", [(4, 2, 64, 64, 32), (3, 1, 20, 12, 8), (2, 2, 9, 7, 4), (5, 5, 32, 96, 32)])
def test_projection_epilogue_with_biases(dtype, H, G, dk, dv, rot):
    """Forms by 16 bytes, by pairs and general, on columns of wider rows."""
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 10 + dk)
    dt, T, page, lead = DT[dtype], 6, 16, 8
    n = H * dk + G * (dk + dv)
    wide = torch.randn(T, lead + n + 8, generator=g, dtype=F).to(dt)
    bias = torch.randn(n, generator=g)
    qw, kw = 1 + 0.3 * torch.randn(dk, generator=g), 1 + 0.3 * torch.randn(dk, generator=g)
    pos = torch.tensor([0, 3, 31, 17, 5, 30])
    m = torch.arange(rot // 2, dtype=F)
    ang = torch.arange(40, dtype=F)[:, None] * 100.0 ** (-2 * m / rot)
    pages = torch.full((4, G, page, dk + dv), float("nan"), dtype=dt, device=dev())
    slots = i32([5, 20, 33, 47, 0, 63])
    q = torch.empty(T, H * dk, dtype=dt, device=dev())
    wd = wide.to(dev())
    ops.masked_qkv_prep(q, wd[:, lead:lead + n], H, G, dk, dv, 1e-5, q_weight=qw.to(dev()), k_weight=kw.to(dev()), cos=ang.cos().float().to(dev()),
                        sin=ang.sin().float().to(dev()), rot=rot, positions=pos.to(torch.int32).to(dev()), pages=pages, slots=slots, page_size=page,
                        bias=bias.to(dev()))
    ops.check_device_errors(dev())
    x = wide[:, lead:lead + n].double() + bias.double()
    wq = plain.turn_pairs(plain.unit_rms(x[:, :H * dk].view(T, H, dk), 1e-5) * qw.double(), pos, rot, 100.0)
    wk = plain.turn_pairs(plain.unit_rms(x[:, H * dk:H * dk + G * dk].view(T, G, dk), 1e-5) * kw.double(), pos, rot, 100.0)
    close(q.view(T, H, dk), wq, TOL[dtype], "queries")
    ent = pages.cpu()[slots.cpu().long() // page, :, slots.cpu().long() % page]           # [T, G, dk + dv]
    close(ent[..., :dk], wk, TOL[dtype], "keys")
    close(ent[..., dk:], x[:, H * dk + G * dk:].view(T, G, dv), TOL[dtype], "values")


@pytest.mark.parametrize("dtype,kernel", [("float32", "general"), ("bfloat16", "general"), ("bfloat16", "portion"), ("bfloat16", "decode")])
@pytest.mark.parametrize("H,G,dk,dv,chunk", [(4, 2, 64, 64, 24), (6, 2, 32, 96, 50), (2, 1, 128, 16, 7)])
def test_attention_inside_chunks_with_a_gate_per_element(dtype, kernel, H, G, dk, dv, chunk):
    """Two requests; one query and key made to stand out in turn at the chunk's first position, at the last one of the chunk before and
    at the query's own."""
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(dk + chunk)
    dt, page, lens = DT[dtype], 16, [chunk * 2 + 3, 41]
    W = 12
    table = torch.full((2, W), -1, dtype=torch.int32)
    order = torch.randperm(2 * W, generator=g)
    pages = torch.full((2 * W, G, page, dk + dv), float("nan"))
    ents = []
    for s, n in enumerate(lens):
        e = torch.randn(n, G, dk + dv, generator=g)
        for j in (n - 1, (n - 1) // chunk * chunk, (n - 1) // chunk * chunk - 1):
            if j >= 0:
                e[j, :, :dk] = 3.0 * e[0, :, :dk].sign()                    # keys that stand out; what they hold tells which was read
                e[j, :, dk:] = 5.0 + j
        e = e.to(dt)
        ents.append(e.double())
        for pg in range((n + page - 1) // page):
            p = int(order[s * W + pg])
            table[s, pg] = p
            m = min(page, n - pg * page)
            pages[p, :, :m] = e[pg * page:pg * page + m].transpose(0, 1).float()
    count = 1 if kernel == "decode" else 5                                  # the last tokens of each request
    T = count * len(lens)
    q = torch.randn(T, H, dk, generator=g)
    for s in range(2):
        q[s * count:(s + 1) * count] = 0.05 * q[s * count:(s + 1) * count] + 0.3 * ents[s][0, :, :dk].sign().float().repeat_interleave(H // G, 0)
    q = q.to(dt)
    gate = torch.randn(T, H * dv + 6, generator=g).to(dt)
    pos = [n - count + i for n in lens for i in range(count)]
    out = torch.full((T, H * dv + 10), float("nan"), dtype=dt, device=dev())
    col = out[:, 4:4 + H * dv]
    gd = gate.to(dev())[:, 2:2 + H * dv]
    args = dict(chunk=chunk, gate=gd, out_scale=0.7)
    qd, pd, td = q.reshape(T, H * dk).to(dev()).contiguous(), pages.to(dt).to(dev()), table.to(dev())
    cu = i32([0, count, 2 * count])
    if kernel == "general":
        ops.attn_masked_general(col, qd, pd, td, i32([0] * count + [1] * count), i32(pos), T, H, G, dk, dv, page, 0.2, **args)
    else:
        single = kernel == "decode"
        scratch = torch.empty(ops.attn_keys_scratch_floats(2, G, dv, 2), dtype=torch.float32, device=dev()) if single else None
        ops.attn_masked_bf16(col, qd, pd, td, cu, i32(pos), 2, ops.attn_keys_tiles([count] * 2, H, G), H, G, dk, dv, page, 0.2, all_single=single,
                             splits=2 if single else 1, scratch=scratch, **args)
    ops.check_device_errors(dev())
    want = torch.zeros(T, H, dv, dtype=F)
    for t in range(T):
        e, p = ents[t // count], pos[t]
        lo = p // chunk * chunk
        for h in range(H):
            kk, vv = e[lo:p + 1, h // (H // G), :dk], e[lo:p + 1, h // (H // G), dk:]
            want[t, h] = torch.softmax(kk @ q[t, h].double() * 0.2, 0) @ vv
    want = want.reshape(T, H * dv) * torch.sigmoid(gate[:, 2:2 + H * dv].double()) * 0.7
    close(col, want, TOL[dtype])
    assert torch.isnan(out[:, :4].float()).all() and torch.isnan(out[:, 4 + H * dv:].float()).all()


# ---- linear attention ---------------------------------------------------------------------------------------------------------------

def _linear_inputs(T, H, dk, dv, dt, seed, lead=0):
    g = torch.Generator().manual_seed(seed)
    packed = torch.randn(T, lead + 2 * H * dk + H * dv, generator=g).to(dt)
    decay = torch.rand(T, H * dk, generator=g) ** 0.05
    decay[:, ::3] = torch.rand(T, (H * dk + 2) // 3, generator=g)           # some channels forget at once
    return packed, decay


def _split(packed, H, dk, dv, lead=0):
    p = packed.double()[:, lead:]
    T = p.shape[0]
    return p[:, :H * dk].view(T, H, dk), p[:, H * dk:2 * H * dk].view(T, H, dk), p[:, 2 * H * dk:].view(T, H, dv)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dk,dv", [(2, 64, 64), (3, 10, 12), (1, 7, 9), (2, 128, 40), (1, 300, 20), (2, 16, 100), (1, 1, 1)])
@pytest.mark.parametrize("chunk", [8, 64, 512])
def test_linear_scan_and_its_chunks(dtype, H, dk, dv, chunk):
    """Three requests in one step (one of them a single token), in chunks of several sizes, then a second step that goes on where the
    states stand; slots nobody owns stay as they were."""
    from cppvllm_b200.csrc import ops
    dt = DT[dtype]
    lens, more = [150, 1, 77], [9, 70, 2]
    seqs = [_linear_inputs(a + b, H, dk, dv, dt, 10 * i + dk, lead=8) for i, (a, b) in enumerate(zip(lens, more))]
    state = torch.full((5, H * dk * dv + 3), 7.0, device=dev())
    slots = [3, 0, 2]
    for s in slots:
        state[s] = 0.0
    want = [plain.linear_scan(q * 0.5, k, v, d.double().view(-1, H, dk)) for (p, d) in seqs for q, k, v in [_split(p, H, dk, dv, 8)]]
    at = [0, 0, 0]
    for step in (lens, more):
        packed = torch.cat([seqs[i][0][at[i]:at[i] + n] for i, n in enumerate(step)]).to(dev())
        gg = torch.cat([seqs[i][1][at[i]:at[i] + n] for i, n in enumerate(step)]).to(dev())
        out = torch.empty(sum(step), H * dv, device=dev())
        cu = i32([0, step[0], step[0] + step[1], sum(step)])
        held = sum(-(-n // chunk) for n in step if n > chunk)
        ends = torch.full((max(1, held * H * dk * dv),), float("nan"), device=dev())
        dec = torch.full((max(1, held * H * dk),), float("nan"), device=dev())
        ops.linear_scan(out, packed, 8, 8 + H * dk, 8 + 2 * H * dk, 0.5, gg, state, cu, i32(slots), step, H, dk, dv, chunk, ends, dec)
        ops.check_device_errors(dev())
        row = 0
        for i, n in enumerate(step):
            close(out[row:row + n].view(n, H, dv), want[i][at[i]:at[i] + n], 2e-5, f"request {i}")
            row += n
            at[i] += n
    assert (state[1] == 7.0).all() and (state[4] == 7.0).all() and (state[0, H * dk * dv:] == 0.0).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dk,dv,rank", [(2, 64, 64, 16), (3, 10, 12, 5), (1, 7, 9, 1), (4, 48, 128, 8), (1, 300, 20, 11), (2, 5, 260, 4)])
def test_linear_step(dtype, H, dk, dv, rank):
    """A step of decoded tokens: low-rank decay, rule, norm, gate and constant in one kernel, against the plain functions, twice."""
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(dk * 7 + dv)
    dt, S, tau, eps, scale = DT[dtype], 3, 6.0, 1e-5, 0.8
    HK, HV = H * dk, H * dv
    n = 2 * HK + 2 * HV + rank
    a2 = torch.randn(HK, rank, generator=g).to(dt)
    ab, nw = torch.randn(HK, generator=g) * 2, 1 + 0.3 * torch.randn(dv, generator=g)
    pitch = (HK // H * HV + 3) // 4 * 4 if dv % 4 == 0 else HK // H * HV
    state = torch.randn(5, pitch, generator=g)
    slots = [4, 1, 2]
    sd = state.to(dev())
    S_ref = [state[s, :H * dk * dv].double().view(H, dk, dv) for s in slots]
    for rep in range(2):
        packed = torch.randn(S, n, generator=g).to(dt)
        out = torch.full((S, HV + 9), float("nan"), dtype=dt, device=dev())
        ops.linear_step(out[:, 5:5 + HV], packed.to(dev()), 0, HK, 2 * HK, 2 * HK + HV, 2 * HK + 2 * HV, a2.to(dev()), ab.to(dev()), dk ** -0.5, tau,
                        nw.to(dev()), eps, scale, sd, i32([0, 1, 2, 3]), i32(slots), S, H, dk, dv)
        ops.check_device_errors(dev())
        p = packed.double()
        z = p[:, 2 * HK + 2 * HV:] @ a2.double().T + ab.double()
        d = plain.channel_decay(z, tau).view(S, H, dk)
        q, k, v = p[:, :HK].view(S, H, dk) * dk ** -0.5, p[:, HK:2 * HK].view(S, H, dk), p[:, 2 * HK:2 * HK + HV].view(S, H, dv)
        gt = p[:, 2 * HK + HV:2 * HK + 2 * HV]
        for s in range(S):
            S_ref[s] = d[s][:, :, None] * S_ref[s] + k[s][:, :, None] * v[s][:, None, :]
            o = torch.einsum("hkv,hk->hv", S_ref[s], q[s])
            want = (plain.unit_rms(o, eps) * nw.double()).reshape(-1) * gt[s] * torch.sigmoid(gt[s]) * scale
            close(out[s, 5:5 + HV], want, TOL[dtype], f"output {s}")
            close(sd[slots[s], :H * dk * dv].view(H, dk, dv), S_ref[s], 2e-5, f"state {s}")
    assert torch.equal(sd[0].cpu(), state[0]) and torch.equal(sd[3].cpu(), state[3])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("groups,G", [(3, 64), (2, 12), (5, 7), (1, 600), (4, 512)])
def test_gated_norm_inside_wider_rows(dtype, groups, G):
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(G)
    dt, T, n = DT[dtype], 5, groups * G
    o, gate, w = torch.randn(T, n, generator=g), torch.randn(T, n + 8, generator=g).to(dt), torch.randn(G, generator=g)
    out = torch.full((T, n + 12), float("nan"), dtype=dt, device=dev())
    ops.gated_norm(out[:, 4:4 + n], o.to(dev()), gate.to(dev())[:, 8:], w.to(dev()), groups, 1e-5, gate_act="silu")
    z = gate[:, 8:].double()
    want = (plain.unit_rms(o.double().view(T, groups, G), 1e-5) * w.double()).reshape(T, n) * z * torch.sigmoid(z)
    close(out[:, 4:4 + n], want, TOL[dtype])
    assert torch.isnan(out[:, :4].float()).all() and torch.isnan(out[:, 4 + n:].float()).all()


# ---- gated recurrence over channels ---------------------------------------------------------------------------------------------------

class Lru:
    """Weights of one layer's recurrence and, per request, inputs and the plain outputs of the whole sequence."""

    def __init__(self, W, parts, taps, dt, lens, seed):
        g = torch.Generator().manual_seed(seed)
        r = lambda *s: torch.randn(*s, generator=g)             # noqa: E731
        part = W // parts
        self.W, self.parts, self.taps, self.dt = W, parts, taps, dt
        self.by, self.bx, self.cb, self.br, self.bi = (r(W) for _ in range(5))
        self.conv, lam = r(W, taps), 3.0 * r(W) - 2.0
        self.gates = (r(parts, 2 * part, part) * part ** -0.5).to(dt)
        self.x = [r(n, 2 * W).to(dt) for n in lens]             # [y | x] projections
        self.nsp = -8.0 * torch.nn.functional.softplus(lam.double())
        w = {"ra": self.gates[:, :part].double(), "ri": self.gates[:, part:].double(), "ra.b": self.br.double().view(parts, part),
             "ri.b": self.bi.double().view(parts, part)}
        rnd = plain.to_bf16 if dt == torch.bfloat16 else plain.identity
        self.want = []
        for x in self.x:
            x = x.double()
            u = rnd(plain.causal_conv(x[:, W:] + self.bx.double(), self.conv.double(), self.cb.double()))
            rr, ii = plain.lru_gates(u, w, "")
            S = plain.lru_scan(plain.lru_log_decay(rr, lam.double()), ii * u)
            self.want.append(S * plain.gelu_tanh(x[:, :W] + self.by.double()))
        d = lambda t: t.float().contiguous().to(dev())          # noqa: E731
        self.d = dict(by=d(self.by), bx=d(self.bx), cb=d(self.cb), br=d(self.br), bi=d(self.bi), conv=d(self.conv.t()), nsp=d(self.nsp),
                      gates=self.gates.to(dev()))

    def state(self, slots):
        return torch.full((slots, self.W * (1 + (self.taps if self.taps > 1 else 0))), 5.0, device=dev())

    def portion(self, rows, q_lens, pos, state, slots, chunk, step=False):
        from cppvllm_b200.csrc import ops
        W, T, d = self.W, sum(q_lens), self.d
        packed = rows.to(dev())
        cu = i32([sum(q_lens[:i]) for i in range(len(q_lens) + 1)])
        out = torch.full((T, W), float("nan"), dtype=self.dt, device=dev())
        if step:
            ops.lru_step(out, packed, 0, W, d["by"], d["bx"], d["conv"], d["cb"], d["gates"], d["br"], d["bi"], d["nsp"], state, cu, i32(slots), i32(pos), T)
        else:
            seq = i32([s for s, n in enumerate(q_lens) for _ in range(n)])
            u = ops.lru_conv(torch.empty(T, W, dtype=self.dt, device=dev()), packed, 0, W, self.parts, d["bx"], d["conv"], d["cb"], state, seq, cu,
                             i32(slots), i32(pos))
            z = ops.lru_gates(torch.empty(T, 2 * W, device=dev()), u, d["gates"])
            chunks = sum(-(-n // chunk) for n in q_lens)
            ops.lru_scan(out, z, u, packed, 0, W, self.parts, self.taps, d["by"], d["bx"], d["br"], d["bi"], d["nsp"], state, cu, i32(slots), i32(pos),
                         q_lens, chunk, torch.full((chunks * 2 * W,), float("nan"), device=dev()))
        ops.check_device_errors(dev())
        return out


SHAPES = [(128, 4, 4), (96, 6, 2), (40, 4, 3), (24, 1, 1), (30, 5, 5), (300, 1, 7), (513, 3, 4), (640, 2, 4)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,parts,taps", SHAPES)
def test_recurrence_in_portions_and_decoded_tokens(dtype, W, parts, taps):
    """Requests of unequal length in one step, cut again and again down to one token, in chunks of several sizes, then tokens one by
    one through the one-kernel form, in slots that held something else before; every output equals the whole sequence's."""
    lens = [150, 33, 90]
    m = Lru(W, parts, taps, DT[dtype], lens, W + taps)
    state, slots = m.state(6), [4, 0, 2]
    for s in slots:
        state[s, :W] = 0.0                                # S starts at zero; inputs before position 0 are zeros by their position
    at = [0, 0, 0]
    steps = [([70, 1, 2], 16), ([2, 3, 60], 32), ([40, 2, 1], 8), ([1, 2, 2], 64), ([3, 20, 3], 1)]
    for q_lens, chunk in steps:
        rows = torch.cat([m.x[i][at[i]:at[i] + n] for i, n in enumerate(q_lens)])
        out = m.portion(rows, q_lens, [at[i] + k for i, n in enumerate(q_lens) for k in range(n)], state, slots, chunk)
        row = 0
        for i, n in enumerate(q_lens):
            close(out[row:row + n], m.want[i][at[i]:at[i] + n], TOL[dtype], f"request {i} from {at[i]}")
            row += n
            at[i] += n
    for k in range(4):                                    # decoded tokens; then the general path takes over once more
        live = [i for i in range(3) if at[i] < lens[i]]
        out = m.portion(torch.cat([m.x[i][at[i]:at[i] + 1] for i in live]), [1] * len(live), [at[i] for i in live], state, [slots[i] for i in live], 32,
                        step=True)
        for r, i in enumerate(live):
            close(out[r], m.want[i][at[i]], TOL[dtype], f"request {i} decoded at {at[i]}")
            at[i] += 1
    n = lens[0] - at[0]
    out = m.portion(m.x[0][at[0]:], [n], list(range(at[0], lens[0])), state, [slots[0]], 16)
    close(out, m.want[0][at[0]:], TOL[dtype], "after decoded tokens")
    assert (state[1] == 5.0).all() and (state[3] == 5.0).all() and (state[5] == 5.0).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("batch", [1, 2, 4, 11, 40])
def test_recurrence_from_the_first_token_decoded(dtype, batch):
    """A batch decoded token by token from position 0, against the whole sequences."""
    m = Lru(96, 3, 4, DT[dtype], [6] * batch, batch)
    state = m.state(batch)
    state[:, :96] = 0.0
    for t in range(6):
        out = m.portion(torch.stack([x[t] for x in m.x]), [1] * batch, [t] * batch, state, list(range(batch))[::-1], 32, step=True)
        close(out, torch.stack([w[t] for w in m.want]), TOL[dtype], f"position {t}")


def test_a_slow_channel_remembers_its_first_token():
    """A decay of 1 - 1e-4 over 3,000 tokens in chunks: what entered first is still there, to float32's rounding."""
    m = Lru(16, 2, 4, torch.float32, [3000], 3)
    lam = torch.full((16,), -9.0, dtype=F)
    m.nsp = -8.0 * torch.nn.functional.softplus(lam)
    m.d["nsp"] = m.nsp.float().to(dev())
    m.x[0][1:, 16:] = 0.0
    m.x[0][0, 16:] = 30.0
    w = {"ra": m.gates[:, :8].double(), "ri": m.gates[:, 8:].double(), "ra.b": m.br.double().view(2, 8), "ri.b": m.bi.double().view(2, 8)}
    x = m.x[0].double()
    u = plain.causal_conv(x[:, 16:] + m.bx.double(), m.conv.double(), m.cb.double())
    r, i = plain.lru_gates(u, w, "")
    want = plain.lru_scan(plain.lru_log_decay(r, lam), i * u) * plain.gelu_tanh(x[:, :16] + m.by.double())
    state = m.state(1)
    state[:, :16] = 0.0
    out = m.portion(m.x[0], [3000], list(range(3000)), state, [0], 128)
    close(out, want, 2e-4)


# ---- feed-forwards --------------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,groups,keep,top,D,T", [(6, 2, 1, 2, 48, 9), (12, 3, 2, 3, 64, 700), (4, 1, 1, 4, 50, 5), (64, 8, 3, 6, 96, 33), (6, 3, 3, 1, 33, 600),
                                                   (9, 9, 4, 4, 128, 513)])
def test_router_with_a_correction_inside_the_best_groups(dtype, E, groups, keep, top, D, T):
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(E * 31 + T)
    x = torch.randn(T, D, generator=g).to(DT[dtype])
    wr = torch.randn(E, D, generator=g) * 0.3
    corr = 0.3 * torch.randn(E, generator=g) - 0.4
    ids = torch.full((T, top), -1, dtype=torch.int32, device=dev())
    wts = torch.full((T, top), float("nan"), device=dev())
    ops.route_topk(ids, wts, x.to(dev()), wr.to(dev()), corr.to(dev()), groups=groups, keep=keep)
    s = torch.softmax(x.double() @ wr.double().T, dim=1)
    want, margin = plain.choose(s, corr.double(), {"top": top, "groups": {"count": groups, "keep": keep}})
    clear = margin > 1e-5
    assert int(clear.sum()) > 0.9 * T
    got = ids.cpu().long()
    assert torch.equal(got[clear].sort(1).values, want[clear].sort(1).values)
    picked = s.gather(1, got)
    close(wts, picked / picked.sum(1, keepdim=True), 1e-5)


@pytest.mark.parametrize("dtype,kernel", [("float32", "rows"), ("bfloat16", "rows"), ("bfloat16", "tcgen05")])
@pytest.mark.parametrize("E,identity,top,D,ff,T", [(5, 1, 2, 48, 24, 7), (8, 4, 3, 96, 32, 200), (3, 3, 1, 64, 40, 130), (2, 1, 3, 72, 16, 3), (4, 0, 2, 40, 8, 20)])
def test_clamped_experts_and_identities(dtype, kernel, E, identity, top, D, ff, T):
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(E * 7 + T)
    dt, limit = DT[dtype], 0.7
    x = torch.randn(T, D, generator=g).to(dt)
    w = {}
    for e in range(E):
        for n, shape in (("gate", (ff, D)), ("up", (ff, D)), ("down", (D, ff))):
            w[f"e{e}.{n}"] = (torch.randn(shape, generator=g) * 2 * shape[1] ** -0.5).to(dt)
    ids = torch.stack([torch.randperm(E + identity, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    if identity:
        ids[0, 0] = E + identity - 1                       # a token whose first choice is an identity
        ids[0, 1:] = torch.arange(top - 1, dtype=torch.int32)
    wts = torch.rand(T, top, generator=g)
    gu = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(E)]).to(dev())
    dn = torch.stack([w[f"e{e}.down"] for e in range(E)]).to(dev())
    y = torch.full((T, D), float("nan"), dtype=dt, device=dev())
    ops.routed_experts(y, x.to(dev()), ids.to(dev()), wts.to(dev()), gu, dn, kernel=kernel, activation="clamped", identity=identity, limit=limit)
    ops.check_device_errors(dev())
    rnd = plain.to_bf16 if dtype == "bfloat16" else plain.identity
    outs = [plain.expert(x.double(), {k: v.double() for k, v in w.items()}, f"e{e}.", limit, rnd) for e in range(E)] + [x.double()] * identity
    outs = torch.stack(outs, 1)                            # [T, E + identity, D]
    want = (outs.gather(1, ids.long()[:, :, None].expand(-1, -1, D)) * wts.double()[:, :, None]).sum(1)
    close(y, want, TOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,I", [(3, 40), (5, 33), (64, 128)])
def test_tanh_gelu_gate(dtype, T, I):
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(I)
    gu = (3 * torch.randn(T, 2 * I, generator=g)).to(DT[dtype])
    out = ops.geglu(torch.empty(T, I, dtype=DT[dtype], device=dev()), gu.to(dev()))
    close(out, plain.gelu_tanh(gu[:, :I].double()) * gu[:, I:].double(), TOL[dtype])


@pytest.mark.parametrize("M,D,I", [(200, 72, 264), (1, 64, 128), (515, 256, 40)])
def test_tanh_gelu_gated_product(M, D, I):
    """The tcgen05 product whose epilogue is the gated activation."""
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(M)
    x, w = torch.randn(M, D, generator=g).to(torch.bfloat16), (torch.randn(2 * I, D, generator=g) * 2 * D ** -0.5).to(torch.bfloat16)
    out = ops.gemm_bf16_tcgen05(torch.empty(M, I, dtype=torch.bfloat16, device=dev()), x.to(dev()), w.to(dev()), geglu=True)
    ops.check_device_errors(dev())
    z = plain.to_bf16(x.double() @ w.double().T)
    close(out, plain.gelu_tanh(z[:, :I]) * z[:, I:], TOL["bfloat16"])
