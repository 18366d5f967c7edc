"""Small Sumevik configurations that differ from one another in every size and option, and a writer of their folders.

          width vocab  layers (mixer; feed-forward)
    sv_a    48    97   pair: chunked 4/2 heads, 16 (8 turned)/24, chunks of 16, beside 3 heads of 10 x 12, tau 8;
                             5 experts + 1 identity in 2 groups, best 1, 2 per token
                       recurrence: 40 channels in 4 parts, 3 taps; dense 56
                       recurrence: 24 channels in 1 part, 1 tap; none
    sv_b    80   131   recurrence: 96 channels in 6 parts, 2 taps; 4 experts, no identity, one group, all 4 per token
                       pair: chunked 6/6 heads, 24 (none turned)/16, chunks of 33, beside 2 heads of 16 x 40, tau 1; dense 100
    sv_c    96   150   recurrence: 128 channels in 4 parts, 4 taps; dense 160
                       pair: chunked 4/2 heads, 64 (32 turned)/64, chunks of 40, beside 2 heads of 32 x 64, tau 20;
                             8 experts + 4 identities in 3 groups, best 2, 3 per token
                       pair: chunked 4/1 heads, 32 (32 turned)/128, chunks of 100, beside 4 heads of 64 x 32, tau 4; none
    sv_d    50    61   pair: chunked 5/5 heads, 10 (4 turned)/6, chunks of 5, beside 1 head of 7 x 9, tau 3;
                             3 experts + 3 identities in 2 groups, both kept, 1 per token
                       recurrence: 30 channels in 5 parts, 5 taps; 2 experts + 1 identity, 3 groups, best 2, 2 per token
    sv_e    64    83   pair: chunked 32/1 heads, 16 (16 turned)/16, chunks of 30, beside 1 head of 300 x 20, tau 16; none
                       pair: chunked 2/1 heads, 160 (6 turned)/144, chunks of 70, beside 3 heads of 130 x 36, tau 12; dense 24
                       recurrence: 300 channels in 1 part, 7 taps; none
Widths of 50 and rows of 10, 6 or 7 elements fit no vector width; sv_b starts with a recurrence, sv_c has the sizes the tensor-core
kernels take, sv_e sizes beyond what the fast kernels take.  Scales, eps, limits, bases and the two output scales all differ."""
import json
import os

import torch


def _pair(left, right, scales):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}}


def _left(heads, kv, dim, vdim, chunk, rot, base, scale):
    m = {"dim": dim, "heads": heads, "kv_heads": kv, "vdim": vdim, "scale": scale, "mask": {"size": chunk}}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
    return m


def _right(heads, dim, vdim, tau, rank):
    return {"dim": dim, "heads": heads, "vdim": vdim, "tau": tau, "a_rank": rank}


def _lru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, identity, groups, keep, top, ff, limit):
    r = {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}
    if identity:
        r["identity"] = identity
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": r}


def _layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def _model(vocab, width, eps, logit_scale, layers):
    return {"architecture": "Sumevik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


SV_A = _model(97, 48, 1e-5, 0.7, [
    _layer(_pair(_left(4, 2, 16, 24, 16, 8, 100.0, 0.3), _right(3, 10, 12, 8.0, 5), (0.6, 1.3)), _moe(5, 1, 2, 1, 2, 24, 0.6)),
    _layer(_lru(40, 4, 3), _dense(56)),
    _layer(_lru(24, 1, 1), None)])
SV_B = _model(131, 80, 1e-6, 1.0, [
    _layer(_lru(96, 6, 2), _moe(4, 0, 1, 1, 4, 16, 1.5)),
    _layer(_pair(_left(6, 6, 24, 16, 33, 0, 0, 0.2), _right(2, 16, 40, 1.0, 3), (1.0, 1.0)), _dense(100))])
SV_C = _model(150, 96, 1e-5, 0.3, [
    _layer(_lru(128, 4, 4), _dense(160)),
    _layer(_pair(_left(4, 2, 64, 64, 40, 32, 10000.0, 0.12), _right(2, 32, 64, 20.0, 8), (0.9, 0.7)), _moe(8, 4, 3, 2, 3, 32, 0.8)),
    _layer(_pair(_left(4, 1, 32, 128, 100, 32, 500.0, 0.18), _right(4, 64, 32, 4.0, 16), (1.2, 0.5)), None)])
SV_D = _model(61, 50, 1e-4, 2.0, [
    _layer(_pair(_left(5, 5, 10, 6, 5, 4, 20.0, 0.4), _right(1, 7, 9, 3.0, 1), (0.5, 0.8)), _moe(3, 3, 2, 2, 1, 12, 0.4)),
    _layer(_lru(30, 5, 5), _moe(2, 1, 3, 2, 2, 20, 1.0))])
SV_E = _model(83, 64, 1e-5, 0.5, [
    _layer(_pair(_left(32, 1, 16, 16, 30, 16, 5000.0, 0.25), _right(1, 300, 20, 16.0, 11), (0.8, 0.9)), None),
    _layer(_pair(_left(2, 1, 160, 144, 70, 6, 1000.0, 0.08), _right(3, 130, 36, 12.0, 4), (1.1, 0.4)), _dense(24)),
    _layer(_lru(300, 1, 7), None)])

# name -> (config, seed, page size)
SETUPS = {"sv_a": (SV_A, 41, 16), "sv_b": (SV_B, 42, 32), "sv_c": (SV_C, 43, 16), "sv_d": (SV_D, 44, 64), "sv_e": (SV_E, 45, 32)}


def write_model(path, cfg, seed, sharpen=3.0):
    """Random weights through the package's random-weights writer (tensor names and shapes come from the architecture), then
    made to show faults: the query norms are scaled up so that attention rests on few keys (an edge that is one token off shows),
    decays of both recurrences spread from fast to slow (a lost state shows far away), biases are large, corrections are mostly
    negative and large (a group left out by 0 instead of minus infinity, or a correction in the weights, shows), routers
    choose with clear margins, and experts' products reach their limits."""
    from cppvllm_b200.weights.random_init import random_tensors
    from cppvllm_b200.weights.safetensors_io import save_safetensors
    import cppvllm_b200.models  # noqa: F401
    os.makedirs(path, exist_ok=True)
    tensors = random_tensors(cfg, seed, std=0.08, norm_spread=0.3)
    for k in list(tensors):
        t = tensors[k].float()
        if k.endswith(".left.q.norm"):
            t = t * sharpen
        elif k.endswith((".q.b", ".k.b", ".v.b", ".y.b", ".x.b", ".conv.b", ".ra.b", ".ri.b")):
            t = t * 5.0
        elif k.endswith(".conv"):
            t = t * 6.0
        elif k.endswith(".lam"):
            t = t * 35.0 - 2.0
        elif k.endswith(".a2.b"):
            t = t * 25.0 + 2.0
        elif k.endswith(".correction"):
            t = t * 3.0 - 0.3
        elif k.endswith(".router"):
            t = t * 4.0
        elif k.endswith((".gate", ".up")) and ".e" in k:
            t = t * 2.0
        elif k == "embed":
            t = t * 4.0
        tensors[k] = t.to(torch.bfloat16)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(os.path.join(path, "model.safetensors"), tensors)
    return path


def random_config(seed, tensor_core=False):
    """A configuration drawn at random: 2 to 5 layers of both kinds in any order, with a dense, a routed or no feed-forward; sizes
    odd, prime, 1 or large; chunks from 1 token to more than a prompt.  With `tensor_core` the attention's key and value sizes are
    multiples of 16, the sizes the tensor-core kernels take."""
    import random
    r = random.Random(3000 + seed)
    width = r.choice([32, 40, 50, 64, 72, 100, 128])
    sizes = [16, 32, 48, 64, 96, 128] if tensor_core else [2, 6, 8, 10, 16, 24, 40, 64]
    layers = []
    for i in range(r.randint(2, 5)):
        if r.random() < 0.5:
            blocks = r.choice([1, 2, 3, 4, 8])
            mixer = _lru(blocks * r.choice([1, 5, 8, 16, 20, 33]), blocks, r.randint(1, 6))
        else:
            kv, group, dim = r.choice([1, 2, 3]), r.choice([1, 2, 4] if tensor_core else [1, 2, 3, 5]), r.choice(sizes)
            left = _left(kv * group, kv, dim, r.choice(sizes), r.choice([1, 2, 7, 32, 64, 300]),
                         r.choice([0] + [x for x in (2, 4, 8, 16, dim) if x <= dim and x % 2 == 0]), r.choice([10.0, 1000.0, 250000.0]),
                         r.choice([0.1, 0.2, 0.35]))
            right = _right(r.choice([1, 2, 3, 5]), r.choice([1, 4, 9, 16, 40, 64, 100]), r.choice([1, 4, 7, 16, 33, 64]),
                           r.choice([1.0, 4.0, 16.0, 30.0]), r.choice([1, 4, 7, 16]))
            mixer = _pair(left, right, (r.choice([0.5, 1.0, 1.4]), r.choice([0.3, 1.0, 1.2])))
        kind = r.random()
        if kind < 0.25:
            mlp = None
        elif kind < 0.55:
            mlp = _dense(r.choice([8, 20, 33, 64]))
        else:
            groups, per = r.choice([1, 2, 3, 4]), r.randint(1, 4)
            keep = r.randint(1, groups)
            identity = r.randint(0, groups * per - 1)
            mlp = _moe(groups * per - identity, identity, groups, keep, r.randint(1, keep * per), r.choice([8, 20, 32]), r.choice([0.5, 1.0, 7.0]))
        layers.append(_layer(mixer, mlp))
    return _model(r.randint(40, 300), width, r.choice([1e-6, 1e-5, 1e-4]), r.choice([0.25, 1.0, 1.7]), layers)


def write_all(base):
    return {name: write_model(os.path.join(base, name), cfg, seed) for name, (cfg, seed, _) in SETUPS.items()}


def page_size(name):
    return SETUPS[name][2]


def config(name):
    return SETUPS[name][0]


def random_tokens(vocab, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


_CLEAR = {}
_REFERENCE = {}


def clear_tokens(model_dir, n, seed, margin=0.01):
    """Random tokens among which no routed feed-forward has a close call: where a decision of the router (between groups, or between
    the last chosen output and the first left out) is taken by less than `margin` in the plain implementation, exact or with 16-bit
    rounding, the token is drawn again.  A model is causal, so a token changes nothing before it and the walk goes from left to
    right.  Another expert changes a token's stream by a large step that later tokens read, and would bury the errors the tests
    look for."""
    import plain_sumevik as plain
    key = (model_dir, n, seed)
    if key in _CLEAR:
        return list(_CLEAR[key])
    cfg, w = plain.read_config(model_dir), plain.read_weights(model_dir)
    toks = random_tokens(cfg["vocab"], n, seed)

    def decides(f):
        r = f["router"]
        return r["top"] < r["experts"] + r.get("identity", 0)
    if not any(l.get("mlp") and l["mlp"]["kind"] == "moe" and decides(l["mlp"]) for l in cfg["layers"]):
        _CLEAR[key] = toks
        return list(toks)

    def smallest(tokens):
        out = None
        for rnd in (plain.identity, plain.to_bf16):
            m = []
            plain.forward_loaded(cfg, w, tokens, rnd=rnd, router_margins=m)
            m = torch.stack(m).min(dim=0).values
            out = m if out is None else torch.minimum(out, m)
        return out

    g = torch.Generator().manual_seed(seed + 7919)
    at = 0
    for _ in range(40 * n):
        m = smallest(toks)
        bad = [i for i in range(at, n) if float(m[i]) < margin]
        if not bad:
            break
        at = bad[0]
        toks[at] = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
    else:
        raise AssertionError(f"no token with a clear routing at position {at}")
    _CLEAR[key] = toks
    return list(toks)


def reference(model_dir, tokens, layer_outputs=None):
    """Logits of one whole sequence from the plain implementation, which reads the folder with its own readers."""
    import plain_sumevik as plain
    if layer_outputs is None:
        key = (model_dir, tuple(tokens))
        if key not in _REFERENCE:
            _REFERENCE[key] = plain.forward(model_dir, tokens)
        return _REFERENCE[key]
    logits, layers = plain.forward(model_dir, tokens, return_layers=True)
    layer_outputs.extend(layers)
    return logits
