"""The kernels that came with Legalix, each alone against float64 arithmetic written here or in tests/plain_legalix.py: the tanh norm with
the residual add, the input of a pass, the projection's epilogue with pairs (i, i + rot / 2), attention behind a window with kept first
tokens and a cap (keys that stand out at every edge, pages given back), latent attention with a sink, the turned parts of latent queries,
the state-space recurrence in all its forms, the gate and norm behind it, and the gated activation on columns of wider rows."""
import math

import pytest
import torch

import plain_legalix as plain

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


# ---- element by element -----------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,D", [(1, 48), (5, 50), (9, 4096), (3, 7)])
@pytest.mark.parametrize("deltas", [0, 1, 2])
def test_tanh_norm_with_the_residual_add(dtype, T, D, deltas):
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(T * D + deltas)
    h, w, b = torch.randn(T, D, generator=g) * 3, torch.randn(D, generator=g), torch.randn(D, generator=g)
    ds = [torch.randn(T, D, generator=g).to(DT[dtype]) for _ in range(deltas)]
    alpha = torch.tensor([0.37])
    hd, out = h.to(dev()), torch.empty(T, D, dtype=DT[dtype], device=dev())
    ops.tanh_update(hd, [x.to(dev()) for x in ds], alpha.to(dev()), w.to(dev()), b.to(dev()), out)
    want = h.double() + sum((x.double() for x in ds), torch.zeros(T, D, dtype=F))
    close(hd, want, 1e-6, "stream")
    close(out, torch.tanh(0.37 * want) * w.double() + b.double(), 2e-6 if dtype == "float32" else 5e-3, "norm")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,D", [(1, 48), (5, 50), (9, 1024)])
@pytest.mark.parametrize("deltas", [0, 1, 2])
def test_the_input_of_a_pass(dtype, T, D, deltas):
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(T + D)
    h, e = torch.randn(T, D, generator=g), torch.randn(T, D, generator=g)
    ds = [torch.randn(T, D, generator=g).to(DT[dtype]) for _ in range(deltas)]
    out = torch.full((T, 2 * D), float("nan"), dtype=DT[dtype], device=dev())
    ops.stream_concat(out, h.to(dev()), [x.to(dev()) for x in ds], e.to(dev()))
    want = torch.cat([h.double() + sum((x.double() for x in ds), torch.zeros(T, D, dtype=F)), e.double()], dim=1)
    close(out, want, 1e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,I,lead", [(5, 64, 16), (3, 33, 5), (70, 40, 8)])
def test_gated_activation_on_columns_of_wider_rows(dtype, T, I, lead):
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(I)
    wide = torch.randn(T, lead + 2 * I + 8, generator=g).to(DT[dtype])
    out = torch.full((T, I + lead), 7.0, dtype=DT[dtype], device=dev())
    ops.geglu(out[:, lead:], wide.to(dev())[:, lead:lead + 2 * I], 0.3)
    x = wide[:, lead:lead + 2 * I].double()
    close(out[:, lead:], 0.3 * plain.gelu_tanh(x[:, :I]) * x[:, I:], 1e-6 if dtype == "float32" else 5e-3)
    assert (out[:, :lead] == 7.0).all()


# ---- attention behind a window that keeps the first tokens ------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,rot,normed", [(4, 2, 64, 64, 32, False), (3, 1, 32, 16, 32, True), (2, 2, 18, 7, 4, False), (2, 1, 48, 48, 12, False),
                                                  (6, 3, 128, 80, 64, False)])
def test_projection_epilogue_with_pairs_across_the_rotation(dtype, H, G, dk, dv, rot, normed):
    """Pairs (i, i + rot / 2): by 16 bytes where half the rotation is whole chunks, element by element elsewhere; with and without norms."""
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 10 + dk)
    dt, T, page, lead = DT[dtype], 6, 16, 8
    n = H * dk + G * (dk + dv)
    wide = torch.randn(T, lead + n + 8, generator=g, dtype=F).to(dt)
    bias = torch.randn(n, generator=g) if normed else None
    qw = 1 + 0.3 * torch.randn(dk, generator=g) if normed else None
    pos = torch.tensor([0, 3, 31, 17, 5, 30])
    ang = torch.arange(40, dtype=F)[:, None] * 100.0 ** (-2 * torch.arange(rot // 2, dtype=F) / rot)
    pages = torch.full((4, G, page, dk + dv), float("nan"), dtype=dt, device=dev())
    slots = i32([5, 20, 33, 47, 0, 63])
    q = torch.empty(T, H * dk, dtype=dt, device=dev())
    put = lambda t: t.to(dev()) if t is not None else None              # noqa: E731
    ops.masked_qkv_prep(q, wide.to(dev())[:, lead:lead + n], H, G, dk, dv, 1e-5, q_weight=put(qw), k_weight=put(qw), cos=ang.cos().float().to(dev()),
                        sin=ang.sin().float().to(dev()), rot=rot, interleaved=False, positions=pos.to(torch.int32).to(dev()), pages=pages, slots=slots,
                        page_size=page, bias=put(bias))
    ops.check_device_errors(dev())
    x = wide[:, lead:lead + n].double() + (bias.double() if normed else 0.0)

    def heads(cols, n_heads):
        y = cols.reshape(T, n_heads, dk)
        return plain.turn(plain.unit_rms(y, 1e-5) * qw.double() if normed else y, pos, rot, 100.0, False)
    close(q.view(T, H, dk), heads(x[:, :H * dk], H), TOL[dtype], "queries")
    ent = pages.cpu()[slots.cpu().long() // page, :, slots.cpu().long() % page]           # [T, G, dk + dv]
    close(ent[..., :dk], heads(x[:, H * dk:H * dk + G * dk], G), TOL[dtype], "keys")
    close(ent[..., dk:], x[:, H * dk + G * dk:].view(T, G, dv), TOL[dtype], "values")


@pytest.mark.parametrize("dtype,kernel", [("float32", "general"), ("bfloat16", "general"), ("bfloat16", "portion"), ("bfloat16", "decode"), ("bfloat16", "split")])
@pytest.mark.parametrize("H,G,dk,dv,window,keep,page", [(4, 2, 64, 64, 24, 5, 16), (6, 2, 32, 96, 70, 20, 32), (2, 1, 128, 80, 7, 100, 16), (16, 1, 16, 16, 1, 1, 32),
                                                        (4, 2, 64, 32, 64, 64, 64), (2, 2, 32, 32, 33, 0, 16)])
def test_attention_behind_a_window_with_kept_first_tokens(dtype, kernel, H, G, dk, dv, window, keep, page):
    """Requests of unequal length whose pages behind the window (but for those of the kept tokens) have been given back: their entries in
    the table are -1 and nothing may read them.  In turn one key stands out at the window's first position, just outside it, at the last
    kept position, just behind it, at the query's own and just behind that."""
    from cppvllm_b200.csrc import ops
    if kernel != "general" and (dk % 16 or dv % 16):
        pytest.skip("sizes of the general kernel")
    g = torch.Generator().manual_seed(dk + window + keep)
    dt, lens, cap, scale = DT[dtype], [259, 65, 3], 6.0, 0.3
    count = 1 if kernel in ("decode", "split") else 3
    W = -(-max(lens) // page)
    S, T = len(lens), count * len(lens)
    base = [torch.randn(n, G, dk + dv, generator=g) * 0.3 for n in lens]
    q = torch.randn(T, H, dk, generator=g) * 0.3
    direction = torch.randn(G, dk, generator=g).sign()
    q = (q + 0.4 * direction.repeat_interleave(H // G, 0)).to(dt)
    pos = [n - count + i for n in lens for i in range(count)]
    order = torch.randperm(S * W, generator=g)
    for place in range(6):
        table = torch.full((S, W), -1, dtype=torch.int32)
        pages = torch.full((S * W, G, page, dk + dv), 0.0)
        ents = []
        for s, n in enumerate(lens):
            e = base[s].clone()
            j = [n - window, n - 1 - window, keep - 1, keep, n - 1, n - 2][place]
            if 0 <= j < n:
                e[j, :, :dk] = direction * 0.8
                e[j, :, dk:] = 5.0
            e = e.to(dt)
            ents.append(e.double())
            first_seen = max(0, n - count - window + 1)
            for pg in range((n + page - 1) // page):
                if (pg + 1) * page <= first_seen and pg * page >= keep:
                    continue                               # given back
                p = int(order[s * W + pg])
                table[s, pg] = p
                m = min(page, n - pg * page)
                pages[p, :, :m] = e[pg * page:pg * page + m].transpose(0, 1).float()
        out = torch.full((T, H * dv + 8), float("nan"), dtype=dt, device=dev())
        col = out[:, 8:]
        qd, pd, td = q.reshape(T, H * dk).to(dev()).contiguous(), pages.to(dt).to(dev()), table.to(dev())
        args = dict(window=window, keep_first=keep, softcap=cap, out_scale=0.7)
        if kernel == "general":
            ops.attn_masked_general(col, qd, pd, td, i32([s for s in range(S) for _ in range(count)]), i32(pos), T, H, G, dk, dv, page, scale, **args)
        else:
            single = kernel != "portion"
            splits = 4 if kernel == "split" else 1
            scratch = torch.empty(ops.attn_keys_scratch_floats(S, G, dv, 4), dtype=torch.float32, device=dev()) if splits > 1 else None
            ops.attn_masked_bf16(col, qd, pd, td, i32([count * s for s in range(S + 1)]), i32(pos), S, ops.attn_keys_tiles([count] * S, H, G), H, G, dk, dv,
                                 page, scale, all_single=single, splits=splits, scratch=scratch, **args)
        ops.check_device_errors(dev())
        want = torch.zeros(T, H, dv, dtype=F)
        for t in range(T):
            e, p = ents[t // count], pos[t]
            vis = plain.window_visible(p + 1, window, keep)[p]
            for h in range(H):
                sc = plain.capped(e[:p + 1, h // (H // G), :dk] @ q[t, h].double() * scale, cap).masked_fill(~vis, -math.inf)
                want[t, h] = torch.softmax(sc, 0) @ e[:p + 1, h // (H // G), dk:]
        close(col, want.reshape(T, H * dv) * 0.7, TOL[dtype], f"place {place}")


# ---- latent attention with a sink ---------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype,kernel", [("float32", "general"), ("bfloat16", "general"), ("bfloat16", "portion"), ("bfloat16", "decode"), ("bfloat16", "split")])
@pytest.mark.parametrize("H,R,dr", [(4, 48, 16), (32, 96, 32), (3, 16, 16)])
def test_latent_attention_with_a_sink(dtype, kernel, H, R, dr):
    """Sinks from far below the scores to far above them; the first token sees itself and the sink alone."""
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(H + R)
    dt, HD, page, lens = DT[dtype], R + dr, 16, [1, 150, 33]
    S, count = len(lens), 1 if kernel in ("decode", "split") else 3
    W = -(-max(lens) // page)
    sink = torch.linspace(-6.0, 12.0, H)
    table, pages, ents = torch.full((S, W), -1, dtype=torch.int32), torch.zeros(S * W, page, HD), []
    order = torch.randperm(S * W, generator=g)
    for s, n in enumerate(lens):
        e = torch.randn(n, HD, generator=g).to(dt)
        ents.append(e.double())
        for pg in range((n + page - 1) // page):
            p = int(order[s * W + pg])
            table[s, pg] = p
            m = min(page, n - pg * page)
            pages[p, :m] = e[pg * page:pg * page + m].float()
    counts = [min(count, n) for n in lens]
    pos = [n - c + i for n, c in zip(lens, counts) for i in range(c)]
    seq = [s for s, c in enumerate(counts) for _ in range(c)]
    T = len(pos)
    q = torch.randn(T, H * HD, generator=g).to(dt)
    out = torch.full((T, H * R), float("nan"), dtype=dt, device=dev())
    qd, pd, td, sd = q.to(dev()), pages.to(dt).to(dev()), table.to(dev()), sink.to(dev())
    if kernel == "general":
        ops.paged_attention_general(out, qd, pd, td, i32(seq), i32(pos), H, 1, HD, page, 0.2, num_tokens=T, keys_are_values=True, value_dim=R, sink=sd,
                                    out_scale=0.6)
    else:
        cu = i32([0] + [sum(counts[:s + 1]) for s in range(S)])
        single, splits = kernel != "portion", 2 if kernel == "split" else 1
        groups = min(n for n in range(1, H + 1) if H % n == 0 and H // n <= 16) if single else 1
        scratch = torch.empty(ops.attn_keys_scratch_floats(S, groups, HD, 2), dtype=torch.float32, device=dev()) if splits > 1 else None
        ops.attn_keys_bf16(out, qd, pd, td, cu, i32(pos), S, S if single else ops.attn_keys_tiles(counts, H, 1), H, groups, HD, page, 0.2, all_single=single,
                           splits=splits, scratch=scratch, value_dim=R, kv_heads_in_pages=1, sink=sd, out_scale=0.6)
    ops.check_device_errors(dev())
    want = torch.zeros(T, H, R, dtype=F)
    for t in range(T):
        e = ents[seq[t]][:pos[t] + 1]
        for h in range(H):
            want[t, h] = plain.sink_softmax((e @ q[t].view(H, HD)[h].double()) * 0.2, sink[h].double()) @ e[:, :R]
    close(out, want.reshape(T, H * R) * 0.6, TOL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,dn,R,dr,rot,dv", [(7, 4, 32, 48, 16, 16, 32), (1, 16, 10, 12, 6, 6, 14), (40, 3, 7, 9, 5, 4, 5)])
def test_products_that_write_to_their_places(dtype, T, H, dn, R, dr, rot, dv):
    """Batched products with results inside wider rows (q_abs in front of the turned part, heads side by side) and the turned parts."""
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(T + H)
    dt = DT[dtype]
    q, uk, uv, o = (torch.randn(*s, generator=g).to(dt) for s in ((T, H * (dn + dr)), (H, dn, R), (H, R, dv), (T, H * R)))
    pos = torch.arange(T) * 3
    ang = torch.arange(3 * T, dtype=F)[:, None] * 50.0 ** (-2 * torch.arange(rot // 2, dtype=F) / rot)
    q_att = torch.full((T, H * (R + dr)), float("nan"), dtype=dt, device=dev())
    qd = q.to(dev())
    torch.bmm(qd.view(T, H, dn + dr)[:, :, :dn].transpose(0, 1), uk.to(dev()), out=q_att.view(T, H, R + dr)[:, :, :R].transpose(0, 1))
    ops.latent_q_turn(q_att, qd, H, dn, R, dr, rot, ang.cos().float().to(dev()), ang.sin().float().to(dev()), pos.to(torch.int32).to(dev()))
    got = q_att.view(T, H, R + dr)
    x = q.double().view(T, H, dn + dr)
    close(got[:, :, :R], torch.einsum("thd,hdr->thr", x[..., :dn], uk.double()), TOL[dtype], "q_abs")
    close(got[:, :, R:], plain.turn(x[..., dn:], pos, rot, 50.0, True), TOL[dtype], "turned part")
    wide = torch.full((T, 8 + H * dv), 3.0, dtype=dt, device=dev())
    torch.bmm(o.to(dev()).view(T, H, R).transpose(0, 1), uv.to(dev()), out=wide[:, 8:].unflatten(1, (H, dv)).transpose(0, 1))
    close(wide[:, 8:], torch.einsum("thr,hrv->thv", o.double().view(T, H, R), uv.double()).reshape(T, H * dv), TOL[dtype], "heads")
    assert (wide[:, :8] == 3.0).all()


# ---- state-space recurrence -----------------------------------------------------------------------------------------------------------

def _mixer(H, G, N, P, taps, parts, dtype, plain_kernels, seed, a_log=None):
    from cppvllm_b200.parts.base import Runtime, Workspace
    from cppvllm_b200.parts.recurrent import StateSpaceMixer
    g = torch.Generator().manual_seed(seed)
    inner, C, D = H * P, H * P + 2 * G * N, 8
    w = {"in": torch.zeros(inner + C + H, D), "conv": torch.randn(C, taps, generator=g) * 0.6, "conv.b": torch.randn(C, generator=g) * 0.3,
         "dt_bias": torch.randn(H, generator=g), "A_log": torch.linspace(-6.0, 2.0, H) if a_log is None else torch.full((H,), a_log),
         "D": 1 + 0.3 * torch.randn(H, generator=g), "norm": 1 + 0.3 * torch.randn(inner, generator=g), "o": torch.zeros(D, inner)}
    rt = Runtime(dev(), DT[dtype], Workspace(dev(), 512, 8), plain_kernels=plain_kernels)
    m = StateSpaceMixer(rt, hidden_size=D, num_heads=H, groups=G, state=N, vdim=P, taps=taps, norm_parts=parts, eps=1e-5)
    m.bind({k: v.to(dev()) for k, v in w.items()})
    return m, {k: v.double() for k, v in w.items()}


def _want(packed, w, H, G, N, P, parts, rnd=plain.identity):
    """From the packed projection of one sequence to the normed rows, times 0.8.  `rnd` rounds what the chunks' products read."""
    T, inner, gn = packed.shape[0], H * P, G * N
    z, u, dt = packed[:, :inner], packed[:, inner:2 * inner + 2 * gn], packed[:, 2 * inner + 2 * gn:]
    u = rnd(plain.silu(plain.causal_conv(u, w["conv"], w["conv.b"])))
    dt = torch.nn.functional.softplus(dt + w["dt_bias"], threshold=60.0)
    y = plain.ssd_scan(u[:, :inner].view(T, H, P), u[:, inner:inner + gn].view(T, G, N), u[:, inner + gn:].view(T, G, N), dt, w["A_log"], w["D"])
    return 0.8 * plain.gated_group_norm(y.reshape(T, inner), z, w["norm"], parts, 1e-5)


def _run(m, state, packed, parts_of, slots):
    """Steps of unequal portions: `parts_of` lists, per step, {sequence: tokens}.  Returns each sequence's rows."""
    from cppvllm_b200.csrc import ops
    from cppvllm_b200.parts.context import StepContext
    at = [0] * len(packed)
    rows = [[] for _ in packed]
    for step in parts_of:
        seqs = sorted(step)
        lens = [step[s] for s in seqs]
        x = torch.cat([packed[s][at[s]:at[s] + n] for s, n in zip(seqs, lens)])
        wide = torch.zeros(x.shape[0], x.shape[1] + 8 + (-x.shape[1]) % 8, dtype=m.rt.dtype, device=dev())
        wide[:, :x.shape[1]] = x.to(dev())
        T = x.shape[0]
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        ctx = StepContext(num_tokens=T, num_seqs=len(seqs), tokens=None, positions=i32([at[s] + i for s, n in zip(seqs, lens) for i in range(n)]),
                          seq_of_token=i32([k for k, n in enumerate(lens) for _ in range(n)]), cu_seqlens=i32(cu), kv_lens=None,
                          state_slots=i32([slots[s] for s in seqs]), groups=[], logit_rows=None, num_logit_rows=0, q_lens=lens,
                          all_decode=all(n == 1 for n in lens))
        out = torch.full((T, m.core_width + 8), float("nan"), dtype=m.rt.dtype, device=dev())
        m.core(wide[:, :x.shape[1]], out[:, :m.core_width], 0.8, ctx, None, state)
        ops.check_device_errors(dev())
        for k, s in enumerate(seqs):
            rows[s].append(out[cu[k]:cu[k + 1], :m.core_width].cpu())
            at[s] += lens[k]
    return [torch.cat(r) for r in rows]


SIZES = [(4, 2, 32, 32, 4, 2), (3, 3, 16, 80, 3, 5), (2, 1, 144, 64, 2, 1), (8, 2, 128, 64, 4, 4), (3, 1, 7, 10, 3, 2), (5, 5, 9, 6, 5, 3), (1, 1, 300, 20, 1, 1),
         (2, 2, 256, 128, 4, 1), (1, 1, 1, 1, 2, 1)]


@pytest.mark.parametrize("dtype,plain_kernels", [("float32", False), ("float32", True), ("bfloat16", False), ("bfloat16", True)])
@pytest.mark.parametrize("H,G,N,P,taps,parts", SIZES)
def test_state_space_mixer_in_every_cutting(dtype, plain_kernels, H, G, N, P, taps, parts):
    """Three sequences in used slots: whole, in portions down to one token across chunk borders, decoded token by token, and mixed."""
    m, w = _mixer(H, G, N, P, taps, parts, dtype, plain_kernels, H + N)
    g = torch.Generator().manual_seed(P + taps)
    lens = [150, 97, 70]
    cols = 2 * H * P + 2 * G * N + H
    packed = [torch.randn(n, cols, generator=g).to(DT[dtype]) for n in lens]
    state = torch.full((5,) + m.state_spec().shape, 3.0, device=dev())       # slots that others have used
    slots = [3, 0, 2]
    state[slots] = 0.0                                                       # as at admission
    want = [_want(p.double(), w, H, G, N, P, parts) for p in packed]
    # where a part's outputs nearly cancel, its norm magnifies the rounding of x, B and C: that much more is allowed there
    slack = [2.0 * (_want(p.double(), w, H, G, N, P, parts, plain.to_bf16) - v).abs() if dtype == "bfloat16" else 0.0 for p, v in zip(packed, want)]

    def near(a, b, s, what):
        over = ((a.double() - b.double()).abs() - slack[s]).max()
        assert float(over) < TOL[dtype] * max(1.0, float(b.abs().max())), f"{what}: {float(over):.2e}"
    cuts = [{0: 64, 1: 2}, {0: 1, 1: 1, 2: 5}, {0: 2, 1: 1, 2: 1}, {0: 1, 1: 1, 2: 1}, {0: 65, 2: 2}, {1: 63, 2: 58}, {0: 1, 1: 1, 2: 1}, {0: 1, 1: 1, 2: 1},
            {0: 15, 1: 26}, {1: 1}, {2: 1}]
    assert [sum(c.get(s, 0) for c in cuts) for s in range(3)] == lens
    got = _run(m, state, packed, cuts, slots)
    assert (state[[1, 4]] == 3.0).all()                                      # nobody else's slot was touched
    for s in range(3):
        near(got[s], want[s], s, f"sequence {s}")
    state[slots] = 0.0
    whole = _run(m, state, packed, [{0: 150, 1: 97, 2: 70}], slots)
    for s in range(3):
        near(whole[s], want[s], s, f"sequence {s} whole")
        near(whole[s], got[s], s, f"sequence {s} cut differently")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decoded_from_the_first_token_at_many_batch_sizes(dtype):
    H, G, N, P, taps, parts = 4, 2, 16, 24, 4, 2
    m, w = _mixer(H, G, N, P, taps, parts, dtype, False, 3)
    g = torch.Generator().manual_seed(5)
    for S in (1, 2, 7):
        packed = [torch.randn(9, 2 * H * P + 2 * G * N + H, generator=g).to(DT[dtype]) for _ in range(S)]
        state = torch.zeros((S + 1,) + m.state_spec().shape, device=dev())
        got = _run(m, state, packed, [{s: 1 for s in range(S)}] * 9, list(range(S)))
        for s in range(S):
            close(got[s], _want(packed[s].double(), w, H, G, N, P, parts), TOL[dtype], f"{S} requests, {s}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_state_that_remembers_its_first_tokens(dtype):
    """Decays of 1 - 1e-5 a token: what the first token of 400 wrote is still there, through chunks, portions and decoded tokens."""
    H, G, N, P, taps, parts = 2, 1, 16, 16, 2, 1
    m, w = _mixer(H, G, N, P, taps, parts, dtype, False, 7, a_log=-11.0)
    g = torch.Generator().manual_seed(9)
    p = torch.randn(400, 2 * H * P + 2 * G * N + H, generator=g) * 0.2
    p[0, H * P:] *= 40.0
    other = p.clone()
    other[0, H * P:] *= -1.0
    p, other = p.to(DT[dtype]), other.to(DT[dtype])
    want, far = _want(p.double(), w, H, G, N, P, parts), _want(other.double(), w, H, G, N, P, parts)
    assert float((want[-1] - far[-1]).abs().max()) > 0.05
    state = torch.zeros((1,) + m.state_spec().shape, device=dev())
    got = _run(m, state, [p], [{0: 200}, {0: 130}, {0: 3}] + [{0: 1}] * 67, [0])
    close(got[0], want, TOL[dtype])


@pytest.mark.parametrize("decay", [-60.0, -1e-6])
def test_chunks_with_decays_at_their_ends(decay):
    """Decays that wipe the state at every token, and decays that change nothing: no overflow, no lost addend."""
    from cppvllm_b200.csrc import ops
    H, G, N, P, T = 2, 1, 32, 32, 200
    g = torch.Generator().manual_seed(2)
    u = torch.randn(T, H * P + 2 * N, generator=g).bfloat16()
    dt, la, skip = torch.rand(T, H, generator=g), torch.full((T, H), decay), torch.randn(H, generator=g)
    la[::7] = -20.0
    state = torch.randn(2, H * N * P, generator=g)
    st = state.to(dev())
    held = ops.ssd_held_chunks(T)
    ends, decays = torch.empty(held * H * N * P, device=dev()), torch.empty(held * H, device=dev())
    y = torch.empty(T, H * P, device=dev())
    ops.ssd_chunks(y, u.to(dev()), dt.to(dev()), la.to(dev()), skip.to(dev()), st, i32([0, T]), i32([1]), [T], H, G, N, P, ends=ends, decays=decays)
    ops.check_device_errors(dev())
    x, B, C = u[:, :H * P].double().view(T, H, P), u[:, H * P:H * P + N].double(), u[:, H * P + N:].double()
    S, want = state[1].double().view(H, N, P), torch.zeros(T, H, P, dtype=F)
    for t in range(T):
        S = torch.exp(la[t].double())[:, None, None] * S + dt[t].double()[:, None, None] * B[t][None, :, None] * x[t][:, None, :]
        want[t] = torch.einsum("hnp,n->hp", S, C[t]) + skip.double()[:, None] * x[t]
    close(y.view(T, H, P), want, 3e-4, "outputs")          # operands are exact: only the split factors' 16 bits round
    close(st[1].view(H, N, P), S, 3e-4, "state")
    assert torch.equal(st[0].cpu(), state[0])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,parts,n", [(3, 2, 96), (1, 3, 10), (5, 1, 4096), (4, 8, 256), (2, 1, 12000), (9, 4, 516)])
def test_gate_and_norm(dtype, T, parts, n):
    from cppvllm_b200.csrc import ops
    g = torch.Generator().manual_seed(n)
    y, z = torch.randn(T, parts * n, generator=g), torch.randn(T, parts * n + 8, generator=g).to(DT[dtype])
    w = 1 + 0.3 * torch.randn(parts * n, generator=g)
    out = torch.full((T, parts * n + 8), 5.0, dtype=DT[dtype], device=dev())
    ops.gate_norm(out[:, 8:], y.to(dev()), z.to(dev())[:, :parts * n], w.to(dev()), parts, 1e-5, 0.4)
    close(out[:, 8:], 0.4 * plain.gated_group_norm(y.double(), z[:, :parts * n].double(), w.double(), parts, 1e-5), 2e-6 if dtype == "float32" else 1e-2)
    assert (out[:, :8] == 5.0).all()


def test_wrappers_refuse_what_the_kernels_cannot_take():
    from cppvllm_b200.csrc import ops
    z = torch.zeros
    d = dev()
    with pytest.raises(ops.KernelError):
        ops.tanh_update(z(2, 4, device=d), (z(2, 5, device=d),), z(1, device=d), z(4, device=d), z(4, device=d), z(2, 4, device=d))
    with pytest.raises(ops.KernelError):
        ops.stream_concat(z(2, 4, device=d), z(2, 4, device=d), (), z(2, 4, device=d))
    with pytest.raises(ops.KernelError):                   # kept first tokens stand beside a window
        ops.attn_masked_general(z(1, 4, device=d), z(1, 4, device=d), z(1, 1, 16, 8, device=d), i32([[0]]), i32([0]), i32([0]), 1, 1, 1, 4, 4, 16, 1.0, keep_first=2)
    with pytest.raises(ops.KernelError):                   # a state of 24 rows is not in steps of 16
        ops.ssd_chunks(z(1, 16, device=d), z(1, 64, device=d, dtype=torch.bfloat16), z(1, 1, device=d), z(1, 1, device=d), z(1, device=d), z(1, 384, device=d),
                       i32([0, 1]), i32([0]), [1], 1, 1, 24, 16)
    with pytest.raises(ops.KernelError):                   # portions of more than a chunk need scratch
        ops.ssd_chunks(z(70, 16, device=d), z(70, 48, device=d, dtype=torch.bfloat16), z(70, 1, device=d), z(70, 1, device=d), z(1, device=d),
                       z(1, 256, device=d), i32([0, 70]), i32([0]), [70], 1, 1, 16, 16)
