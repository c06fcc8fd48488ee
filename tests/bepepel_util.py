"""Tiny Bepepel configurations, weights and model folders for the tests.  The list of tensors
comes from the plain implementation (not from the package's builder), the weights are drawn with
torch's generator and written with the package's safetensors writer."""
import copy
import json
import os

import torch

import plain_bepepel as plain


def gla(heads, dim, vdim, tau=8.0, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def left(heads, kv_heads, dim, vdim, conv, window=None, keep=0, rot=None, base=10000.0, bands=None, scale=None):
    """``rot``: turned dimensions (None: nothing turns); ``bands`` = (factor, low, high, original)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
         "scale": scale if scale is not None else dim ** -0.5}
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot is not None:
        m["rot"] = {"dims": rot, "base": base}
        if bands:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    return m


def right(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def parallel(a, b, scales=(1.0, 1.0), mlp=None):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": a, "right": b, "left_scale": scales[0], "right_scale": scales[1]}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def model(width, vocab, layers, eps=1e-6, mult=0.6, logit_scale=0.5):
    return {"architecture": "Bepepel", "vocab": vocab, "width": width, "residual_mult": mult, "logit_scale": logit_scale,
            "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # both mixers and feed-forwards, a window shorter than two pages and no multiple of one, one layer that
    # sees everything, turns nothing and has single taps, a layer without feed-forward, with and without a
    # shared expert
    "mix": dict(config=model(64, 160, [
        parallel(left(4, 2, 16, 8, conv=4, window=20, keep=3, rot=8, bands=(3.0, 1.0, 3.0, 64)),
                 right(4, 16, 24, groups=2, conv=2, norm_groups=4), (0.7, 1.4), mlp=moe(6, 3, 24, shared=40)),
        gla(4, 16, 8, mlp=dense(96)),
        gla(2, 24, 20, tau=3.0, mlp=None),
        parallel(left(6, 1, 8, 12, conv=1), right(2, 24, 16, groups=1, conv=1, norm_groups=1), (1.3, 0.8), mlp=moe(4, 1, 16)),
    ]), seed=51, page_size=16, rank=16),
    # nothing a multiple of 8, one query head per key head, every dimension turned, more kept keys than a page
    # has room for, two taps beside five, a group for every head, a rank that is no multiple of 4
    "odd": dict(config=model(52, 211, [
        gla(3, 6, 10, tau=20.0, mlp=moe(9, 2, 14, shared=10)),
        parallel(left(5, 5, 6, 10, conv=2, window=9, keep=11, rot=6, base=300.0, bands=(1.5, 0.5, 2.0, 20), scale=0.6),
                 right(3, 5, 7, groups=3, conv=5, norm_groups=5), (1.1, 0.9), mlp=dense(30)),
        parallel(left(2, 1, 10, 6, conv=5, window=33, keep=1, rot=4), right(4, 7, 9, groups=2, conv=3, norm_groups=2),
                 (0.5, 0.6), mlp=None),
    ], eps=3e-6, mult=1.0, logit_scale=1.0), seed=52, page_size=8, rank=5),
    # sizes the tensor-core kernels take: a window of exactly two pages with kept keys beyond a key tile of the
    # attention kernel, values wider than keys, states of 64 to 160 rows, every expert chosen in one layer
    "wide": dict(config=model(256, 384, [
        gla(2, 128, 96, tau=16.0, mlp=moe(16, 4, 128, shared=256)),
        parallel(left(8, 2, 64, 128, conv=4, window=64, keep=70, rot=32, bands=(8.0, 1.0, 4.0, 128)),
                 right(8, 32, 64, groups=4, conv=4, norm_groups=2), (0.8, 1.1), mlp=dense(512)),
        parallel(left(4, 1, 16, 32, conv=3, window=100, keep=2, rot=16), right(16, 16, 160, groups=2, conv=4, norm_groups=8),
                 (1.2, 0.7), mlp=moe(4, 4, 32)),
        gla(4, 64, 64, tau=4.0, mlp=moe(8, 2, 64, shared=64)),
    ], mult=0.4, logit_scale=0.2), seed=53, page_size=32, rank=24),
    # windows of hundreds of positions (many pages and key tiles; single tokens' keys cut into shares)
    "long": dict(config=model(128, 200, [
        parallel(left(4, 2, 32, 32, conv=4, window=300, keep=20, rot=16, bands=(4.0, 1.0, 4.0, 128)),
                 right(4, 32, 48, groups=1, conv=4, norm_groups=1), mlp=dense(128)),
        gla(2, 48, 32, mlp=moe(4, 2, 32, shared=32)),
        parallel(left(2, 2, 32, 48, conv=2, window=512, keep=5, rot=32), right(8, 8, 32, groups=8, conv=3, norm_groups=4), mlp=None),
    ]), seed=54, page_size=16, rank=8),
}


def random_weights(config, seed, rank=16):
    """Weights as float32 tensors holding bfloat16 values."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in plain.tensor_shapes(config, rank).items():
        last = name.split(".")[-1]
        t = torch.randn(shape, generator=g)
        if last in ("norm1", "norm2", "norm", "D"):
            t = 1.0 + 0.2 * t
        elif name.endswith("a2.b"):
            t = 1.0 + t
        elif last == "A_log":
            t = 0.7 * t - 1.0
        elif last == "dt_bias":
            t = t - 1.0
        elif last == "b":
            t = 0.3 * t
        elif last == "conv":
            t = t / shape[-1] ** 0.5
        elif last != "embed":
            t = t / shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16).float()
    return out


def sharpen(config, weights):
    """Makes far keys, kept first keys and the edges of windows matter (scores grow, so that every softmax
    falls on one or two of the visible keys), and what happened long ago (decays close to 1)."""
    config, out = copy.deepcopy(config), dict(weights)
    for e in config["layers"]:
        if e["type"] == "parallel":
            e["mixer"]["left"]["scale"] *= 10.0
    for name, t in weights.items():
        if name.endswith("a2.b"):
            out[name] = (t + 4.0).to(torch.bfloat16).float()
        elif name.endswith("A_log"):
            out[name] = (t - 4.0).to(torch.bfloat16).float()
    return config, out


def make_folder(folder, name, sharp=False):
    """Writes config.json and model.safetensors (bfloat16); returns (config, weights as float32)."""
    from dispec_b200.weights import write_safetensors

    spec = CONFIGS[name]
    config = copy.deepcopy(spec["config"])
    weights = random_weights(config, spec["seed"], spec["rank"])
    if sharp:
        config, weights = sharpen(config, weights)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    write_safetensors(os.path.join(folder, "model.safetensors"),
                      {k: v.to(torch.bfloat16) for k, v in weights.items()})
    return config, weights
