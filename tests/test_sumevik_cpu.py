"""The plain Sumevik implementation against closed forms, the test models against the faults they are made to show, and the
configuration reader's refusals.  No GPU."""
import copy
import math

import pytest
import torch

import plain_sumevik as plain
import sumevik_models as sm

F = torch.float64


@pytest.fixture(scope="module")
def sv_dirs(tmp_path_factory):
    return sm.write_all(str(tmp_path_factory.mktemp("sumevik_cpu")))


def test_convolution_looks_back_and_starts_from_zeros():
    p = torch.arange(1.0, 6.0, dtype=F)[:, None]
    y = plain.causal_conv(p, torch.tensor([[100.0, 10.0, 1.0]], dtype=F), torch.tensor([0.5], dtype=F))
    assert y.flatten().tolist() == [1.5, 12.5, 123.5, 234.5, 345.5]


def test_gated_recurrence_in_closed_form():
    """Gates at 1/2: l = -4 softplus(lam); a constant input c gives S_t = sqrt(1 - a^2) c / 2 (1 + a + .. + a^t)."""
    lam = torch.tensor([0.3, -4.0], dtype=F)
    w = {"ra": torch.zeros(1, 2, 2, dtype=F), "ri": torch.zeros(1, 2, 2, dtype=F), "ra.b": torch.zeros(1, 2, dtype=F), "ri.b": torch.zeros(1, 2, dtype=F)}
    u = torch.ones(6, 2, dtype=F) * torch.tensor([2.0, -3.0], dtype=F)
    r, i = plain.lru_gates(u, w, "")
    S = plain.lru_scan(plain.lru_log_decay(r, lam), i * u)
    a = torch.exp(-4.0 * torch.log1p(torch.exp(lam)))
    for t in range(6):
        want = torch.sqrt(1 - a * a) * 0.5 * u[0] * sum(a ** k for k in range(t + 1))
        assert torch.allclose(S[t], want)


def test_gate_matrices_belong_to_their_part():
    w = {"ra": torch.stack([torch.eye(2, dtype=F), 2 * torch.eye(2, dtype=F)]), "ri": torch.zeros(2, 2, 2, dtype=F),
         "ra.b": torch.zeros(2, 2, dtype=F), "ri.b": torch.zeros(2, 2, dtype=F)}
    w["ra"][0, 0, 1] = 5.0                                # row = output
    u = torch.tensor([[1.0, 0.1, 0.3, -0.2]], dtype=F)
    r, _ = plain.lru_gates(u, w, "")
    assert torch.allclose(r[0], torch.sigmoid(torch.tensor([1.5, 0.1, 0.6, -0.4], dtype=F)))


def test_linear_attention_is_a_decayed_sum():
    g = torch.Generator().manual_seed(1)
    q, k = torch.randn(5, 2, 3, generator=g, dtype=F), torch.randn(5, 2, 3, generator=g, dtype=F)
    v, d = torch.randn(5, 2, 4, generator=g, dtype=F), torch.rand(5, 2, 3, generator=g, dtype=F)
    o = plain.linear_scan(q, k, v, d)
    for h in range(2):
        want = torch.zeros(4, dtype=F)
        for j in range(5):
            decay = torch.ones(3, dtype=F)
            for m in range(j + 1, 5):
                decay = decay * d[m, h]
            want = want + (q[4, h] * decay * k[j, h]).sum() * v[j, h]
        assert torch.allclose(o[4, h], want)
    assert torch.allclose(plain.channel_decay(torch.tensor([0.0, 50.0], dtype=F), 2.0), torch.tensor([math.sqrt(0.5), 1.0], dtype=F))


def test_chunks_and_rotation():
    c = plain.chunk_visible(12, 5)
    assert c[4, 0] and c[4, 4] and not c[5, 4] and c[5, 5] and c[9, 5] and not c[10, 9] and not c[3, 4]
    one = plain.turn_pairs(torch.tensor([[1.0, 0.0, 1.0, 0.0, 7.0]], dtype=F), torch.tensor([3]), 4, 100.0)
    assert torch.allclose(one, torch.tensor([[math.cos(3.0), math.sin(3.0), math.cos(0.3), math.sin(0.3), 7.0]], dtype=F))


def test_choice_by_groups_with_a_correction():
    s = torch.tensor([[0.4, 0.1, 0.2, 0.05, 0.15, 0.1]], dtype=F)
    router = {"experts": 4, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 1}}
    ids, m = plain.choose(s, torch.tensor([-1.0, -1.0, -1.0, -1.0, -0.5, -0.9], dtype=F), router)
    # all choice scores are negative; the last group's best (0.15 - 0.5) wins, so both its outputs are chosen
    assert sorted(ids[0].tolist()) == [4, 5] and abs(float(m[0]) - 0.25) < 1e-12
    router["groups"]["keep"] = 2
    ids, _ = plain.choose(s, torch.zeros(6, dtype=F), router)
    assert ids[0].tolist() == [0, 2]
    h = torch.tensor([[2.0, -1.0]], dtype=F)
    w = {"router": torch.zeros(6, 2, dtype=F), "correction": torch.tensor([-1.0, -1.0, -1.0, -1.0, 1.0, 1.0], dtype=F)}
    y = plain.routed_experts(h, w, "", {"expert": {"limit": 1.0}, "router": dict(router, groups={"count": 3, "keep": 1})})
    assert torch.allclose(y, h)                           # two identity experts whose weights add up to 1


def test_clamped_experts():
    w = {"e.gate": torch.tensor([[3.0], [-3.0]], dtype=F), "e.up": torch.tensor([[-9.0], [0.5]], dtype=F), "e.down": torch.eye(2, dtype=F)}
    y = plain.expert(torch.ones(1, 1, dtype=F), w, "e.", 2.0)
    sg = lambda z: 1.0 / (1.0 + math.exp(-z))             # noqa: E731
    want = [2.0 * sg(1.702 * 2.0) * (-2.0 + 1.0), -3.0 * sg(1.702 * -3.0) * 1.5]      # the gate has no lower limit
    assert torch.allclose(y[0], torch.tensor(want, dtype=F))


FAULTS = ["chunk", "state", "lru_state", "conv_state", "bias", "gate", "correction_in_weights", "zero_for_other_groups", "identity",
          "limit", "left_scale", "logit_scale", "tau"]


@pytest.mark.parametrize("fault", FAULTS)
def test_the_test_models_show_the_faults_they_are_made_for(sv_dirs, monkeypatch, fault):
    """A chunk's edge that is one token off, a state or a convolution's history lost at a cut, a bias or a gate left out, a correction
    that enters the weights, groups left out by 0, identity experts left out, a limit or a constant ignored: each moves the logits by
    far more than the tolerance."""
    d = sv_dirs["sv_a"]
    toks = sm.clear_tokens(d, 90, 1)
    good = plain.forward(d, toks)
    cfg, w = plain.read_config(d), plain.read_weights(d)
    patch = lambda name, fn: monkeypatch.setattr(plain, name, fn)       # noqa: E731
    cut = 45                                              # where a portion would begin
    if fault == "chunk":
        patch("chunk_visible", lambda T, size: (torch.arange(T)[None, :] <= torch.arange(T)[:, None])
              & ((torch.arange(T)[:, None] + 1) // size == (torch.arange(T)[None, :] + 1) // size))
    elif fault == "state":
        scan = plain.linear_scan
        patch("linear_scan", lambda q, k, v, g: torch.cat([scan(q[:cut], k[:cut], v[:cut], g[:cut]), scan(q[cut:], k[cut:], v[cut:], g[cut:])]))
    elif fault == "lru_state":
        lru = plain.lru_scan
        patch("lru_scan", lambda a, x: torch.cat([lru(a[:cut], x[:cut]), lru(a[cut:], x[cut:])]))
    elif fault == "conv_state":
        conv = plain.causal_conv
        patch("causal_conv", lambda p, c, b: torch.cat([conv(p[:cut], c, b), conv(p[cut:], c, b)]))
    elif fault == "bias":
        w = {k: (torch.zeros_like(v) if k.endswith(".left.v.b") else v) for k, v in w.items()}
    elif fault == "gate":
        w = {k: (torch.zeros_like(v) if k.endswith(".left.g") else v) for k, v in w.items()}
    elif fault == "correction_in_weights":
        choose = plain.choose

        def routed(h, w, p, f, rnd=plain.identity, margins=None):
            s = torch.softmax(h @ w[p + "router"].T, dim=1) + w[p + "correction"]
            ids, _ = choose(s, torch.zeros_like(w[p + "correction"]), f["router"])
            picked = s.gather(1, ids)
            wt = picked / picked.sum(1, keepdim=True)
            y = torch.zeros_like(h)
            for t in range(h.shape[0]):
                for c, e in enumerate(ids[t].tolist()):
                    y[t] += wt[t, c] * (plain.expert(h[t:t + 1], w, f"{p}e{e}.", f["expert"]["limit"])[0] if e < f["router"]["experts"] else h[t])
            return y
        patch("routed_experts", routed)
    elif fault == "zero_for_other_groups":
        def choose(s, correction, router):
            c = s + correction
            g = router["groups"]
            best = c.view(len(c), g["count"], -1).max(2).values
            keep = torch.zeros_like(best, dtype=torch.bool).scatter_(1, best.topk(g["keep"], dim=1).indices, True)
            c = c.masked_fill(~keep.repeat_interleave(c.shape[1] // g["count"], dim=1), 0.0)
            return c.topk(router["top"], dim=1).indices, torch.zeros(len(c), dtype=F)
        patch("choose", choose)
    elif fault == "identity":
        cfg["layers"][0]["mlp"]["router"]["experts"] = 6
        w.update({f"l0.mlp.e5.{n}": torch.zeros_like(w[f"l0.mlp.e0.{n}"]) for n in ("gate", "up", "down")})
    elif fault == "limit":
        cfg["layers"][0]["mlp"]["expert"]["limit"] = 1e9
    elif fault == "left_scale":
        cfg["layers"][0]["mixer"]["left_scale"] = 1.0
    elif fault == "logit_scale":
        cfg["logit_scale"] = 1.0
    elif fault == "tau":
        cfg["layers"][0]["mixer"]["right"]["tau"] = 1.0
    bad = plain.forward_loaded(cfg, w, toks)
    moved = float((bad - good).abs().max()) / float(good.abs().max())
    assert moved > 1e-2, f"{fault}: the logits moved by {moved:.2e} of their size only"


def test_configuration_reader():
    from cppvllm_b200.config.model_config import ConfigError
    from cppvllm_b200.config.registry import resolve_architecture
    from cppvllm_b200.config.sumevik_config import SumevikConfig
    cfg = SumevikConfig.from_dict(sm.SV_A)
    m, f = cfg.layers[0].mixer, cfg.layers[0].mlp
    assert (m.left.heads, m.left.kv_heads, m.left.chunk, m.left.rot_dims, m.right.tau, m.left_scale, m.right_scale) == (4, 2, 16, 8, 8.0, 0.6, 1.3)
    assert (f.experts, f.identity, f.groups, f.keep, f.top, f.limit) == (5, 1, 2, 1, 2, 0.6)
    assert cfg.layers[1].mixer.blocks == 4 and cfg.layers[1].mlp.kind == "dense" and cfg.layers[2].mlp is None and cfg.logit_scale == 0.7
    assert SumevikConfig.from_dict(sm.SV_B).layers[1].mixer.left.rot_dims == 0 and SumevikConfig.from_dict(sm.SV_B).layers[0].mlp.identity == 0
    assert resolve_architecture(sm.SV_A).name == "Sumevik"

    def broken(change):
        d = copy.deepcopy(sm.SV_A)
        change(d)
        with pytest.raises(ConfigError):
            SumevikConfig.from_dict(d)
    pair, moe = lambda d: d["layers"][0]["mixer"], lambda d: d["layers"][0]["mlp"]          # noqa: E731
    broken(lambda d: d["layers"][0].update(type="serial"))
    broken(lambda d: d.update(layers=[]))
    broken(lambda d: d.pop("vocab"))
    broken(lambda d: pair(d).pop("left"))
    broken(lambda d: pair(d).pop("right_scale"))
    broken(lambda d: pair(d)["left"].update(kv_heads=3))
    broken(lambda d: pair(d)["left"]["rot"].update(dims=7))
    broken(lambda d: pair(d)["left"]["rot"].update(dims=18))
    broken(lambda d: pair(d)["right"].update(tau=0))
    broken(lambda d: d["layers"][1]["mixer"].update(blocks=3))
    broken(lambda d: d["layers"][1]["mixer"].pop("conv"))
    broken(lambda d: d["layers"][1]["mlp"].update(kind="sparse"))
    broken(lambda d: moe(d)["expert"].pop("limit"))
    broken(lambda d: moe(d)["router"].update(identity=2))                 # seven outputs in two groups
    broken(lambda d: moe(d)["router"].update(top=4))                      # more than the kept group holds
    broken(lambda d: moe(d)["router"]["groups"].pop("keep"))


def test_the_model_as_data_names_every_tensor():
    from cppvllm_b200.weights.random_init import random_tensors
    t = random_tensors(sm.SV_A, 1)
    assert t["l0.norm1"].shape == (48,) and t["final.norm"].shape == (48,) and t["embed"].shape == (97, 48) and "head" not in t
    assert t["l0.mix.left.q"].shape == (64, 48) and t["l0.mix.left.k.b"].shape == (32,) and t["l0.mix.left.v"].shape == (48, 48)
    assert t["l0.mix.left.g"].shape == (96, 48) and t["l0.mix.left.o"].shape == (48, 96) and t["l0.mix.left.k.norm"].shape == (16,)
    assert t["l0.mix.right.q"].shape == (30, 48) and t["l0.mix.right.v"].shape == (36, 48) and t["l0.mix.right.norm"].shape == (12,)
    assert t["l0.mix.right.a2"].shape[0] == 30 and t["l0.mix.right.a2.b"].shape == (30,) and t["l0.mix.right.o"].shape == (48, 36)
    assert t["l0.mlp.router"].shape == (6, 48) and t["l0.mlp.correction"].shape == (6,) and t["l0.mlp.e4.down"].shape == (48, 24)
    assert "l0.mlp.e5.gate" not in t and "l0.mlp.shared.gate" not in t and "l2.norm2" not in t
    assert t["l1.mix.ra"].shape == (4, 10, 10) and t["l1.mix.ri.b"].shape == (4, 10) and t["l1.mix.conv"].shape == (40, 3)
    assert t["l1.mix.lam"].shape == (40,) and t["l1.mlp.down"].shape == (48, 56) and t["l2.mix.conv"].shape == (24, 1)


def test_members_of_a_pair_keep_one_cache_and_one_state():
    from cppvllm_b200.config.registry import resolve_architecture
    from cppvllm_b200.parts.base import Runtime, Workspace
    from cppvllm_b200.parts.model import CausalLM
    from cppvllm_b200.parts.side_by_side import SideBySideMixer
    arch = resolve_architecture(sm.SV_A)
    cpu = torch.device("cpu")
    model = CausalLM(arch.build_spec(arch.parse_config(sm.SV_A)), Runtime(cpu, torch.float32, Workspace(cpu, 0), max_positions=8))
    specs = model.state_specs()
    assert [s.shape for s in specs] == [(3 * 10 * 12,), (40 * 4,), (24,)] and list(model.cache_units()) == [0]
    assert model.cache_units()[0].entry_shape == (2, 40)
    pair = model.blocks[0].mixer
    with pytest.raises(ValueError):
        SideBySideMixer(model.rt, hidden_size=48, members=[pair.members[0], pair.members[0]], scales=(1.0, 1.0))
    with pytest.raises(ValueError):
        SideBySideMixer(model.rt, hidden_size=48, members=[pair.members[0], pair.members[1]], scales=(1.0,))


@pytest.mark.parametrize("T,q_lens", [(1, [1]), (64, [64]), (300, [300]), (2048, [2048]), (4000, [1, 3000, 999]), (8192, [4096, 4096])])
def test_chunk_scratch_is_large_enough(T, q_lens):
    """The buffers that are sized once for the largest step hold the chunks of every smaller one."""
    from cppvllm_b200.csrc import ops
    for H, dk, dv in ((1, 4, 8), (6, 48, 64), (16, 64, 128), (64, 300, 256)):
        n = ops.linear_chunk_tokens(T, H, dk, dv)
        held = sum(c for c in (-(-q // n) for q in q_lens) if c > 1)
        assert n % 8 == 0 and held <= ops.linear_held_chunks(max(T, 64), H, dk, dv) and held <= ops.linear_held_chunks(8192, H, dk, dv)
    for W in (24, 160, 1024, 4096):
        n = ops.lru_chunk_tokens(T, W)
        assert sum(-(-q // n) for q in q_lens) <= ops.lru_most_chunks(8192, len(q_lens), W)
