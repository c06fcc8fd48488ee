"""Tiny Pikalorn configurations, weights and model folders for the tests.  The list of tensors
comes from the plain implementation (not from the package's builder), the weights are drawn with
torch's generator and written with the package's safetensors writer."""
import copy
import json
import os

import torch

import plain_pikalorn as plain


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, base=10000.0, slowed=None, scale=None, kv_from=None, ff=None, dims=None):
    """``slowed`` = (factor, original, fast, slow); ``dims``: turned dimensions (None: all of rot_dim)."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "scale": scale if scale is not None else (dim + rot_dim) ** -0.5,
         "rot": {"dims": rot_dim if dims is None else dims, "base": base}}
    if slowed:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), slowed))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": dense(ff)}


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "delta", "mlp": dense(ff),
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attention(heads, kv_heads, dim, rot=None, base=10000.0, scale=None, ff=None):
    return {"type": "attention", "mlp": dense(ff),
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim,
                      "scale": scale if scale is not None else dim ** -0.5,
                      "rot": {"dims": dim if rot is None else rot, "base": base}}}


def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def model(width, vocab, layers, eps=1e-6, scale=3.0):
    return {"architecture": "Pikalorn", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": layers}


CONFIGS = {
    # every mixer, with and without feed-forward, latents read by two later layers (one of them behind layers of
    # other kinds), slowed and plain rotation, partly turned heads, groups of one to four heads
    "mix": dict(config=model(64, 160, [
        delta(4, 2, 16, 24, conv=4, ff=96),
        latent(4, 16, 16, 8, 32, 24, slowed=(4.0, 64, 32.0, 1.0), ff=64),
        attention(4, 2, 16, rot=8, ff=128),
        latent(6, 8, 16, 16, 32, 40, slowed=(4.0, 64, 32.0, 1.0), kv_from=1, ff=48),
        delta(3, 3, 8, 16, conv=2),
        attention(6, 6, 8),
        latent(2, 24, 16, 12, 32, 16, slowed=(4.0, 64, 32.0, 1.0), kv_from=1),
        latent(3, 8, 8, 8, 48, 20, base=500.0, ff=80),
    ]), seed=61, page_size=16),
    # nothing a multiple of 8, single taps, one head in a group of five, heads that are not turned at all or only in
    # two dimensions, a feed-forward no kernel fuses
    "odd": dict(config=model(52, 211, [
        latent(5, 6, 10, 7, 18, 14, base=300.0, slowed=(1.5, 20, 4.0, 0.5), scale=0.31, dims=6, ff=30),
        delta(3, 1, 5, 7, conv=1, ff=23),
        delta(5, 5, 10, 6, conv=5),
        attention(5, 1, 10, rot=2, base=77.0, scale=0.4, ff=17),
        latent(3, 5, 10, 9, 18, 11, base=300.0, slowed=(1.5, 20, 4.0, 0.5), scale=0.5, dims=6, kv_from=0, ff=34),
        attention(4, 2, 6, rot=0, scale=0.7),
    ], eps=3e-5, scale=1.0), seed=62, page_size=8),
    # sizes the tensor-core kernels take: latents of 64 to 320, states of 33 to 200 rows, wide groups
    "wide": dict(config=model(256, 384, [
        latent(8, 32, 32, 64, 80, 96, base=1e5, slowed=(16.0, 128, 16.0, 2.0), ff=512),
        delta(4, 2, 128, 96, conv=4, ff=256),
        attention(8, 1, 64, rot=32, ff=384),
        latent(16, 64, 32, 32, 80, 64, base=1e5, slowed=(16.0, 128, 16.0, 2.0), kv_from=0, ff=128),
        delta(2, 2, 200, 32, conv=3, ff=64),
        attention(2, 2, 128, ff=64),
        latent(2, 16, 16, 128, 320, 48, ff=96),
        delta(4, 1, 33, 20, conv=2, ff=32),
    ]), seed=63, page_size=32),
    # contexts of hundreds of tokens (single tokens' keys cut into shares, many pages)
    "long": dict(config=model(128, 200, [
        latent(4, 32, 16, 32, 112, 64, slowed=(8.0, 256, 32.0, 1.0), ff=128),
        delta(4, 2, 48, 32, conv=4, ff=128),
        attention(4, 2, 32, rot=16),
        latent(4, 16, 16, 16, 112, 32, slowed=(8.0, 256, 32.0, 1.0), kv_from=0, ff=64),
    ]), seed=64, page_size=16),
}


def random_weights(config, seed):
    """Weights as float32 tensors holding bfloat16 values."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in plain.tensor_shapes(config).items():
        last = name.split(".")[-1]
        t = torch.randn(shape, generator=g)
        if last in ("norm1", "norm"):
            t = 1.0 + 0.2 * t
        elif last == "A_log":
            t = 0.7 * t - 1.0
        elif last == "dt_bias":
            t = t - 1.0
        elif last == "sink":
            t = 1.5 * t + 1.0
        elif last == "b" and len(shape) == 1:  # biases (the gate projection of a delta layer has that name too)
            t = 0.3 * t
        elif last != "embed":
            t = t / shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16).float()
    return out


def sharpen(config, weights):
    """Makes far keys matter (scores grow, so that every softmax falls on one or two of the keys or the sink) and
    what happened long ago (decays close to 1)."""
    config, out = copy.deepcopy(config), dict(weights)
    for e in config["layers"]:
        if e["type"] != "delta":
            e["mixer"]["scale"] *= 8.0
    for name, t in weights.items():
        if name.endswith("A_log"):
            out[name] = (t - 4.0).to(torch.bfloat16).float()
        elif name.endswith("sink"):
            out[name] = (t * 3.0).to(torch.bfloat16).float()
    return config, out


def make_folder(folder, name, sharp=False):
    """Writes config.json and model.safetensors (bfloat16); returns (config, weights as float32)."""
    from dispec_b200.weights import write_safetensors

    spec = CONFIGS[name]
    config = copy.deepcopy(spec["config"])
    weights = random_weights(config, spec["seed"])
    if sharp:
        config, weights = sharpen(config, weights)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in weights.items()})
    return config, weights
