"""The plain Legalix implementation against closed forms, the test models against the faults they are made to show, and the
configuration reader's refusals.  No GPU."""
import copy
import math

import pytest
import torch

import legalix_models as lm
import plain_legalix as plain

F = torch.float64


@pytest.fixture(scope="module")
def lg_dirs(tmp_path_factory):
    return lm.write_all(str(tmp_path_factory.mktemp("legalix_cpu")))


def test_dynamic_tanh():
    w = {"n": torch.tensor([2.0, 3.0], dtype=F), "n.b": torch.tensor([0.5, -1.0], dtype=F), "n.alpha": torch.tensor(0.25, dtype=F)}
    y = plain.dynamic_tanh(torch.tensor([[4.0, -8.0]], dtype=F), w, "n")
    assert torch.allclose(y, torch.tensor([[2 * math.tanh(1.0) + 0.5, -3 * math.tanh(2.0) - 1.0]], dtype=F))


def test_rotation_in_both_layouts():
    x, p = torch.tensor([[1.0, 0.0, 0.0, 1.0, 7.0]], dtype=F), torch.tensor([3])
    pairs = plain.turn(x, p, 4, 100.0, True)              # (0, 1) by 3, (2, 3) by 0.3
    assert torch.allclose(pairs, torch.tensor([[math.cos(3.0), math.sin(3.0), -math.sin(0.3), math.cos(0.3), 7.0]], dtype=F))
    halves = plain.turn(x, p, 4, 100.0, False)            # (0, 2) by 3, (1, 3) by 0.3
    assert torch.allclose(halves, torch.tensor([[math.cos(3.0), -math.sin(0.3), math.sin(3.0), math.cos(0.3), 7.0]], dtype=F))


def test_window_with_kept_first_tokens():
    v = plain.window_visible(12, 4, 2)
    assert v[9, 6] and not v[9, 5] and v[9, 0] and v[9, 1] and not v[9, 2] and v[9, 9] and not v[8, 9] and v[3, 0] and v[5, 2] and not v[6, 2]
    none = plain.window_visible(5, 1, 0)
    assert torch.equal(none, torch.eye(5, dtype=torch.bool))


def test_sink_and_cap():
    s = torch.tensor([[1.0, -math.inf, 2.0]], dtype=F)
    a = plain.sink_softmax(s, torch.tensor(0.5, dtype=F))
    total = math.exp(1.0) + math.exp(2.0) + math.exp(0.5)
    assert torch.allclose(a, torch.tensor([[math.exp(1.0) / total, 0.0, math.exp(2.0) / total]], dtype=F))
    assert abs(float(plain.capped(torch.tensor(1e4, dtype=F), 5.0)) - 5.0) < 1e-9 and abs(float(plain.capped(torch.tensor(0.01, dtype=F), 5.0)) - 0.01) < 1e-6


def test_convolution_looks_back_and_starts_from_zeros():
    p = torch.arange(1.0, 6.0, dtype=F)[:, None]
    y = plain.causal_conv(p, torch.tensor([[100.0, 10.0, 1.0]], dtype=F), torch.tensor([0.5], dtype=F))
    assert y.flatten().tolist() == [1.5, 12.5, 123.5, 234.5, 345.5]


def test_state_space_recurrence_is_a_decayed_sum():
    g = torch.Generator().manual_seed(1)
    T, H, G, N, P = 6, 4, 2, 3, 5
    x, B, C = torch.randn(T, H, P, generator=g, dtype=F), torch.randn(T, G, N, generator=g, dtype=F), torch.randn(T, G, N, generator=g, dtype=F)
    dt, a_log, D = torch.rand(T, H, generator=g, dtype=F), torch.randn(H, generator=g, dtype=F), torch.randn(H, generator=g, dtype=F)
    y = plain.ssd_scan(x, B, C, dt, a_log, D)
    for h in range(H):
        want = D[h] * x[5, h]
        for s in range(T):
            want = want + (C[5, h // 2] @ B[s, h // 2]) * math.exp(-math.exp(a_log[h]) * float(dt[s + 1:, h].sum())) * dt[s, h] * x[s, h]
        assert torch.allclose(y[5, h], want)


def test_gate_comes_before_the_norm_of_each_part():
    y, z = torch.tensor([[3.0, 4.0, 1.0, 1.0]], dtype=F), torch.tensor([[50.0, 50.0, 50.0, 100.0]], dtype=F)      # silu(z) = z out there
    got = plain.gated_group_norm(y, z, torch.tensor([1.0, 1.0, 2.0, 2.0], dtype=F), 2, 0.0)
    a, b = math.sqrt(12.5), math.sqrt(2.5)
    assert torch.allclose(got, torch.tensor([[3 / a, 4 / a, 2 / b, 4 / b]], dtype=F))


def test_layers_in_a_loop():
    cfg = {"layers": [{}] * 5, "loop": {"start": 1, "stop": 3, "times": 2}}
    assert plain.run_order(cfg) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False), (4, False)]
    assert plain.run_order({"layers": [{}] * 2}) == [(0, False), (1, False)]


FAULTS = ["window", "kept", "kept_too_many", "sink", "cap", "mult", "state", "conv_state", "loop_input", "loop_once", "second_input", "dt_bias", "skip",
          "gate_behind_norm", "norm_parts", "pairing", "embedding_scale", "shift", "group"]


@pytest.mark.parametrize("fault", FAULTS)
def test_the_test_models_show_the_faults_they_are_made_for(lg_dirs, monkeypatch, fault):
    """A window or the kept tokens one off, a sink, a cap or a constant left out, a state or a convolution's history lost at a cut, the
    embedding output left out of a pass's input, a pass left out, and so on: each moves the logits by far more than the tolerance."""
    d = lg_dirs["lg_a"]
    toks = lm.tokens(d, 90, 1)
    good = plain.forward(d, toks)
    cfg, w = plain.read_config(d), plain.read_weights(d)
    patch = lambda name, fn: monkeypatch.setattr(plain, name, fn)       # noqa: E731
    cut = 45                                              # where a portion would begin
    mask = cfg["layers"][1]["mixer"]["mask"]
    if fault == "window":
        mask["size"] += 1
    elif fault == "kept":
        mask["keep_first"] -= 1
    elif fault == "kept_too_many":
        mask["keep_first"] += 1
    elif fault == "sink":
        patch("sink_softmax", lambda s, sink: torch.softmax(s, dim=-1))
    elif fault == "cap":
        patch("capped", lambda s, cap: s)
    elif fault == "mult":
        cfg["residual_mult"] = 1.0
    elif fault == "state":
        scan = plain.ssd_scan
        patch("ssd_scan", lambda x, B, C, dt, a, D: torch.cat([scan(x[:cut], B[:cut], C[:cut], dt[:cut], a, D), scan(x[cut:], B[cut:], C[cut:], dt[cut:], a, D)]))
    elif fault == "conv_state":
        conv = plain.causal_conv
        patch("causal_conv", lambda p, c, b: torch.cat([conv(p[:cut], c, b), conv(p[cut:], c, b)]))
    elif fault == "loop_input":
        patch("pass_input", lambda x, x0, w, rnd=None: torch.cat([x, torch.zeros_like(x0)], dim=1) @ w["loop.in"].T)
    elif fault == "loop_once":
        cfg["loop"]["times"] = 1
    elif fault == "second_input":                         # the second pass begins without a product of its own
        order = plain.run_order(cfg)
        patch("run_order", lambda c: order[:3] + [(i, False) for i, _ in order[3:]])
    elif fault == "dt_bias":
        w = {k: (torch.zeros_like(v) if k.endswith(".dt_bias") else v) for k, v in w.items()}
    elif fault == "skip":
        w = {k: (torch.zeros_like(v) if k.endswith(".mix.D") else v) for k, v in w.items()}
    elif fault == "gate_behind_norm":
        patch("gated_group_norm", lambda y, z, wt, n, eps: plain.unit_rms(y.view(len(y), n, -1), eps).reshape(y.shape) * wt * plain.silu(z))
    elif fault == "norm_parts":
        cfg["layers"][0]["mixer"]["norm_groups"] = 1
    elif fault == "pairing":
        turn = plain.turn
        patch("turn", lambda x, p, dims, base, inter: turn(x, p, dims, base, not inter))
    elif fault == "embedding_scale":
        cfg["embedding"]["scale"] = 1.0
    elif fault == "shift":
        w = {k: (torch.zeros_like(v) if k.endswith(".norm1.b") else v) for k, v in w.items()}
    elif fault == "group":                                # the second group's heads read the first group's B and C
        scan = plain.ssd_scan
        patch("ssd_scan", lambda x, B, C, dt, a, D: scan(x, B[:, :1], C[:, :1], dt, a, D))
    bad = plain.forward_loaded(cfg, w, toks)
    moved = float((bad - good).abs().max()) / float(good.abs().max())
    assert moved > 1e-2, f"{fault}: the logits moved by {moved:.2e} of their size only"


def test_configuration_reader():
    from cppvllm_b200.config.legalix_config import LegalixConfig
    from cppvllm_b200.config.model_config import ConfigError
    from cppvllm_b200.config.registry import resolve_architecture
    cfg = LegalixConfig.from_dict(lm.LG_A)
    s, a, l = (cfg.layers[i].mixer for i in range(3))
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first, a.softcap, a.rot_dims, a.scale) == (4, 2, 16, 24, 12, 3, 4.0, 8, 0.3)
    assert (l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.rot_dims) == (3, 10, 6, 14, 9, 12, 6)
    assert (s.heads, s.state, s.vdim, s.groups, s.conv, s.norm_groups) == (3, 7, 10, 1, 3, 2)
    assert [x.ff for x in cfg.layers] == [56, 40, 0, 0] and (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == (1, 3, 2)
    assert cfg.residual_mult == 0.7 and cfg.embedding_scale == 3.0 and LegalixConfig.from_dict(lm.LG_C).loop is None
    assert resolve_architecture(lm.LG_A).name == "Legalix"
    bare = copy.deepcopy(lm.LG_A)
    for k in ("embedding", "residual_mult", "loop"):
        bare.pop(k)
    for k in ("mask", "softcap", "rot", "kv_heads", "vdim"):
        bare["layers"][1]["mixer"].pop(k)
    bare["layers"][2]["mixer"].pop("q_rank")
    b = LegalixConfig.from_dict(bare)
    assert (b.embedding_scale, b.residual_mult, b.layers[1].mixer.window, b.layers[1].mixer.softcap, b.layers[1].mixer.kv_heads, b.layers[1].mixer.vdim,
            b.layers[2].mixer.q_rank) == (1.0, 1.0, 0, 0.0, 4, 16, -1)

    def broken(change):
        d = copy.deepcopy(lm.LG_A)
        change(d)
        with pytest.raises(ConfigError):
            LegalixConfig.from_dict(d)
    m = lambda d, i: d["layers"][i]["mixer"]              # noqa: E731
    broken(lambda d: d["layers"][0].update(type="mamba"))
    broken(lambda d: d.update(layers=[]))
    broken(lambda d: d.pop("vocab"))
    broken(lambda d: d["layers"][0].pop("mixer"))
    broken(lambda d: m(d, 0).update(groups=2))
    broken(lambda d: m(d, 0).update(norm_groups=4))
    broken(lambda d: m(d, 0).pop("conv"))
    broken(lambda d: m(d, 1).update(kv_heads=3))
    broken(lambda d: m(d, 1)["mask"].pop("size"))
    broken(lambda d: m(d, 1)["mask"].update(keep_first=-1))
    broken(lambda d: m(d, 1)["rot"].update(dims=7))
    broken(lambda d: m(d, 1)["rot"].update(dims=18))
    broken(lambda d: m(d, 1).pop("scale"))
    broken(lambda d: m(d, 2).pop("rot"))
    broken(lambda d: m(d, 2)["rot"].update(dims=8))
    broken(lambda d: m(d, 2).update(kv_rank=0))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="moe"))
    broken(lambda d: d["layers"][0]["mlp"].update(ff=0))
    broken(lambda d: d["loop"].update(stop=5))
    broken(lambda d: d["loop"].update(start=3))
    broken(lambda d: d["loop"].update(times=0))


def _model(cfg):
    from cppvllm_b200.config.registry import resolve_architecture
    from cppvllm_b200.parts.base import Runtime, Workspace
    from cppvllm_b200.parts.model import CausalLM
    arch, cpu = resolve_architecture(cfg), torch.device("cpu")
    return CausalLM(arch.build_spec(arch.parse_config(cfg)), Runtime(cpu, torch.float32, Workspace(cpu, 0), max_positions=8))


def test_the_model_as_data_names_every_tensor():
    from cppvllm_b200.weights.random_init import random_tensors
    t = random_tensors(lm.LG_A, 1)
    want = {"embed": (97, 48), "head": (97, 48), "loop.in": (48, 96), "final.norm": (48,), "final.norm.b": (48,), "final.norm.alpha": (),
            "l0.norm1": (48,), "l0.norm1.b": (48,), "l0.norm1.alpha": (), "l0.mix.in": (30 + 44 + 3, 48), "l0.mix.conv": (44, 3), "l0.mix.conv.b": (44,),
            "l0.mix.dt_bias": (3,), "l0.mix.A_log": (3,), "l0.mix.D": (3,), "l0.mix.norm": (30,), "l0.mix.o": (48, 30),
            "l0.mlp.gate": (56, 48), "l0.mlp.up": (56, 48), "l0.mlp.down": (48, 56),
            "l1.mix.q": (64, 48), "l1.mix.k": (32, 48), "l1.mix.v": (48, 48), "l1.mix.o": (48, 96), "l1.mlp.gate": (40, 48),
            "l2.mix.dq": (9, 48), "l2.mix.dq.norm": (9,), "l2.mix.uq": (48, 9), "l2.mix.dkv": (18, 48), "l2.mix.dkv.norm": (12,), "l2.mix.uk": (30, 12),
            "l2.mix.uv": (42, 12), "l2.mix.sink": (3,), "l2.mix.o": (48, 42), "l3.mix.conv": (32 + 2 * 2 * 12, 2)}
    for name, shape in want.items():
        assert tuple(t[name].shape) == shape, name
    assert not any(n.startswith(("l2.mlp", "l3.mlp")) or n.endswith((".norm2", ".g", ".q.norm")) for n in t)


def test_every_pass_has_its_own_cache_and_state():
    m = _model(lm.LG_A)
    assert [(e.layer, e.input) for e in m.run_order] == [(0, None), (1, "loop"), (2, None), (1, "loop"), (2, None), (3, None)]
    units = m.cache_units()
    assert len(units) == 4 and len({e.cache for e in m.run_order}) == 6
    window = [c for c in units.values() if c.window]
    assert len(window) == 2 and all((c.window, c.keep_first, c.entry_shape) == (12, 3, (2, 40)) for c in window)
    assert [c.entry_shape for c in units.values() if not c.window] == [(18,), (18,)]
    sizes = [s.shape[0] if s is not None else 0 for s in m.state_specs()]
    assert sizes == [-(-(3 * 7 * 10 + 3 * 44) // 4) * 4, 0, 0, 0, 0, 4 * 12 * 8 + 2 * 80] and all(s % 4 == 0 for s in sizes)
    twice = _model(lm.LG_E)                               # a loop that reaches the end, over a layer with a state
    assert [(e.layer, e.input) for e in twice.run_order] == [(0, None), (1, "loop"), (2, None), (1, "loop"), (2, None)]
    assert [s is not None for s in twice.state_specs()] == [False, False, True, False, True]


def test_mixer_and_feed_forward_share_their_products():
    m = _model(lm.LG_A)
    group = m.blocks[0].mixer
    assert [type(x).__name__ for x in group.members] == ["StateSpaceMixer", "GatedMLP"] and group.scales == (0.7, 0.7) and group.core_width == 30 + 56
    t = {n: torch.zeros(ws.shape) for n, ws in m.weight_specs().items()}
    group.bind(t)
    # every member's rows start on whole 16-byte pieces of bf16 outputs: 77 rows take 80
    assert group.w_in.shape == (80 + 112, 48) and group.in_cols == [(0, 77), (80, 192)] and group.w_o.shape == (48, 86)
    assert len(m.blocks[2].mixer.members) == 1            # a layer without a feed-forward


def test_parts_refuse_sizes_that_contradict_one_another():
    from cppvllm_b200.parts.attention_masked import MaskedAttention
    from cppvllm_b200.parts.recurrent import StateSpaceMixer
    rt = _model(lm.LG_A).rt
    with pytest.raises(ValueError):
        MaskedAttention(rt, hidden_size=8, num_heads=2, num_kv_heads=1, dim=4, vdim=4, scale=1.0, eps=1e-5, keep_first=3)     # kept tokens need a window
    ok = dict(hidden_size=8, num_heads=2, groups=1, state=4, vdim=4, taps=2, norm_parts=2, eps=1e-5)
    for bad in (dict(groups=3), dict(norm_parts=3), dict(taps=0), dict(state=513)):
        with pytest.raises(ValueError):
            StateSpaceMixer(rt, **dict(ok, **bad))


@pytest.mark.parametrize("q_lens", [[1], [64], [65], [2048], [1, 3000, 999], [4096, 4096], [65] * 120, [130] * 63])
def test_chunk_scratch_is_large_enough(q_lens):
    """The buffers that are sized once for the largest step hold the chunks of every smaller one."""
    from cppvllm_b200.csrc import ops
    held = sum(c for c in (-(-q // ops.SSD_CHUNK) for q in q_lens) if c > 1)
    assert held <= ops.ssd_held_chunks(max(sum(q_lens), 64)) and held <= ops.ssd_held_chunks(8192)
