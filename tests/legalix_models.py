"""Small Legalix configurations that differ from one another in every size and option, and a writer of their folders.

          width vocab  layers (mixer; feed-forward)
    lg_a    48    97   recurrence: 3 heads of 7 x 10, 1 group, 3 taps, norm in 2 parts; 56
                       attention: 4/2 heads, 16 (8 turned)/24, window of 12, 3 kept, cap 4; 40
                       latent: 3 heads, 10 + 6, values of 14, latents of 9 and 12; none
                       recurrence: 4 heads of 12 x 8, 2 groups, 2 taps, norm in 1 part; none          layers 1 .. 2 run twice
    lg_b    96   131   attention: 4/2 heads, 64 (32 turned)/32, window of 40, 20 kept, cap 6; 160
                       recurrence: 4 heads of 32 x 32, 2 groups, 4 taps, norm in 4 parts; 96
                       latent: 4 heads, 32 + 16, values of 32, latents of 40 and 48; 64               layers 0 .. 2 run three times
    lg_c   128   150   recurrence: 3 heads of 144 x 80, 3 groups, 4 taps, norm in 5 parts; 128
                       latent: 32 heads, 16 + 16, values of 16, latents of 64 and 96; 128
                       attention: 8/1 heads, 128 (128 turned)/16, window of 16, 70 kept, cap 9; 112   no loop
    lg_d    50    61   latent: 5 heads, 3 + 4, values of 6, latents of 7 and 11; 33
                       attention: 5/5 heads, 10 (4 turned)/7, window of 1, none kept, cap 2; none
                       recurrence: 5 heads of 9 x 6, 5 groups, 5 taps, norm in 3 parts; 20            layer 1 runs once (its input is there)
    lg_e    64    83   attention: 2/1 heads, 160 (160 turned)/144, window of 70, 5 kept, cap 30; 24
                       latent: 2 heads, 40 + 24, values of 36, latents of 50 and 200; 48
                       recurrence: 1 head of 300 x 20, 1 group, 1 tap, norm in 1 part; 60             layers 1 .. 2 run twice, to the end
Widths of 50 and rows of 10, 7 or 6 elements fit no vector width, and lg_d's norm parts cross its heads; lg_b and lg_c have sizes the
tensor-core kernels take, lg_e sizes beyond what the fast kernels take.  Scales, eps, caps, bases and multipliers all differ."""
import json
import os

import torch


def _attention(heads, kv, dim, vdim, window, keep, rot, base, scale, cap):
    return {"type": "attention", "mixer": {"dim": dim, "heads": heads, "kv_heads": kv, "vdim": vdim, "scale": scale, "softcap": cap,
                                           "mask": {"size": window, "keep_first": keep}, "rot": {"dims": rot, "base": base}}}


def _latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base, scale):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                  "scale": scale, "rot": {"dims": rot_dim, "base": base}}}


def _ssd(heads, state, vdim, groups, conv, parts):
    return {"type": "mamba2", "mixer": {"heads": heads, "state": state, "vdim": vdim, "groups": groups, "conv": conv, "norm_groups": parts}}


def _layer(mixer, ff):
    return dict(mixer, mlp={"kind": "dense", "ff": ff} if ff else None)


def _model(vocab, width, eps, embedding, mult, layers, loop=None):
    c = {"architecture": "Legalix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embedding}, "residual_mult": mult,
         "layers": layers}
    if loop is not None:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


LG_A = _model(97, 48, 1e-5, 3.0, 0.7, [
    _layer(_ssd(3, 7, 10, 1, 3, 2), 56),
    _layer(_attention(4, 2, 16, 24, 12, 3, 8, 100.0, 0.3, 4.0), 40),
    _layer(_latent(3, 10, 6, 14, 9, 12, 50.0, 0.35), 0),
    _layer(_ssd(4, 12, 8, 2, 2, 1), 0)], (1, 3, 2))
LG_B = _model(131, 96, 1e-6, 5.0, 0.4, [
    _layer(_attention(4, 2, 64, 32, 40, 20, 32, 10000.0, 0.1, 6.0), 160),
    _layer(_ssd(4, 32, 32, 2, 4, 4), 96),
    _layer(_latent(4, 32, 16, 32, 40, 48, 300.0, 0.16), 64)], (0, 3, 3))
LG_C = _model(150, 128, 1e-5, 2.0, 0.5, [
    _layer(_ssd(3, 144, 80, 3, 4, 5), 128),
    _layer(_latent(32, 16, 16, 16, 64, 96, 2000.0, 0.2), 128),
    _layer(_attention(8, 1, 128, 16, 16, 70, 128, 500.0, 0.05, 9.0), 112)])
LG_D = _model(61, 50, 1e-4, 4.0, 1.2, [
    _layer(_latent(5, 3, 4, 6, 7, 11, 20.0, 0.5), 33),
    _layer(_attention(5, 5, 10, 7, 1, 0, 4, 30.0, 0.4, 2.0), 0),
    _layer(_ssd(5, 9, 6, 5, 5, 3), 20)], (1, 2, 1))
LG_E = _model(83, 64, 1e-5, 1.5, 0.6, [
    _layer(_attention(2, 1, 160, 144, 70, 5, 160, 1000.0, 0.05, 30.0), 24),
    _layer(_latent(2, 40, 24, 36, 50, 200, 5000.0, 0.12), 48),
    _layer(_ssd(1, 300, 20, 1, 1, 1), 60)], (1, 3, 2))

# name -> (config, seed, page size)
SETUPS = {"lg_a": (LG_A, 51, 16), "lg_b": (LG_B, 52, 32), "lg_c": (LG_C, 53, 16), "lg_d": (LG_D, 54, 64), "lg_e": (LG_E, 55, 32)}


def write_model(path, cfg, seed, sharpen=2.5):
    """Random weights through the package's random-weights writer (tensor names and shapes come from the architecture), then made to
    show faults: queries and keys are scaled up so that attention rests on few keys (an edge that is one token off shows) and scores
    reach the cap, sinks are large, decays spread from fast to slow (a lost state shows far away), biases are large."""
    from cppvllm_b200.weights.random_init import random_tensors
    from cppvllm_b200.weights.safetensors_io import save_safetensors
    import cppvllm_b200.models  # noqa: F401
    os.makedirs(path, exist_ok=True)
    tensors = random_tensors(cfg, seed, std=0.08, norm_spread=0.3)
    for k in list(tensors):
        t = tensors[k].float()
        if k.endswith((".mix.q", ".mix.k", ".mix.uq", ".mix.uk")):
            t = t * sharpen
        elif k.endswith(".sink"):
            t = t * 20.0
        elif k.endswith((".norm1.b", ".norm.b", ".conv.b")):
            t = t * 4.0
        elif k.endswith(".conv"):
            t = t * 6.0
        elif k.endswith(".A_log"):
            t = t * 20.0 - 2.0
        elif k.endswith(".dt_bias"):
            t = t * 12.0
        elif k == "embed":
            t = t * 5.0
        tensors[k] = t.to(torch.bfloat16)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(os.path.join(path, "model.safetensors"), tensors)
    return path


def random_config(seed, tensor_core=False):
    """A configuration drawn at random: 1 to 5 layers of the three kinds in any order, with or without a feed-forward, with or without a
    loop over any of them; sizes odd, prime, 1 or large; windows from 1 token to more than a prompt.  With `tensor_core` the sizes are
    the ones the tensor-core kernels take."""
    import random
    r = random.Random(4000 + seed)
    width = r.choice([32, 40, 50, 64, 72, 100, 128])
    sizes = [16, 32, 48, 64, 96, 128] if tensor_core else [1, 2, 6, 7, 8, 10, 16, 24, 40, 64]
    layers = []
    for i in range(r.randint(1, 5)):
        kind = r.choice(["attention", "latent", "ssd"])
        if kind == "attention":
            kv, group, dim = r.choice([1, 2, 3]), r.choice([1, 2, 4] if tensor_core else [1, 2, 3, 5]), r.choice([s for s in sizes if s > 1])
            mixer = _attention(kv * group, kv, dim, r.choice(sizes), r.choice([1, 2, 7, 32, 64, 300]), r.choice([0, 1, 4, 33, 64, 100]),
                               r.choice([x for x in (2, 4, 8, 16, dim) if x <= dim and x % 2 == 0]), r.choice([10.0, 1000.0, 250000.0]),
                               r.choice([0.05, 0.1, 0.2]), r.choice([1.0, 5.0, 50.0]))
        elif kind == "latent":
            rot = r.choice([16, 32] if tensor_core else [2, 4, 10, 24])
            rank = r.choice([16, 48, 96] if tensor_core else [1, 5, 12, 40, 130])
            mixer = _latent(r.choice([1, 2, 3, 5, 20]), r.choice(sizes), rot, r.choice(sizes), r.choice([1, 7, 24, 40]), rank, r.choice([10.0, 10000.0]),
                            r.choice([0.1, 0.2, 0.35]))
        else:
            groups = r.choice([1, 2, 3])
            heads, vdim = groups * r.choice([1, 2, 4]), r.choice(sizes)
            parts = r.choice([p for p in range(1, 9) if heads * vdim % p == 0])
            mixer = _ssd(heads, r.choice(sizes), vdim, groups, r.randint(1, 6), parts)
        layers.append(_layer(mixer, r.choice([0, 8, 20, 33, 64])))
    loop = None
    if r.random() < 0.7:
        a = r.randint(0, len(layers) - 1)
        loop = (a, r.randint(a + 1, len(layers)), r.choice([1, 2, 3]))
    return _model(r.randint(40, 300), width, r.choice([1e-6, 1e-5, 1e-4]), r.choice([1.0, 3.0, 6.0]), r.choice([0.3, 0.6, 1.0]), layers, loop)


def write_all(base):
    return {name: write_model(os.path.join(base, name), cfg, seed) for name, (cfg, seed, _) in SETUPS.items()}


def page_size(name):
    return SETUPS[name][2]


def config(name):
    return SETUPS[name][0]


def tokens(model_dir, n, seed):
    with open(os.path.join(model_dir, "config.json")) as f:
        vocab = json.load(f)["vocab"]
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


_REFERENCE = {}


def reference(model_dir, toks, layer_outputs=None):
    """Logits of one whole sequence from the plain implementation, which reads the folder with its own readers."""
    import plain_legalix as plain
    if layer_outputs is None:
        key = (model_dir, tuple(toks))
        if key not in _REFERENCE:
            _REFERENCE[key] = plain.forward(model_dir, toks)
        return _REFERENCE[key]
    logits, layers = plain.forward(model_dir, toks, return_layers=True)
    layer_outputs.extend(layers)
    return logits
