"""Tiny Nidorax configurations and weights for the tests.

The configurations differ from each other in every size and constant and include the corner values: one head, one expert
chosen and all of them, one group and as many groups as experts, every group kept, decays of zero and one, key, value and
latent sizes that differ, one turning pair and no scaling of the frequencies, cached rows narrower and wider than the
tensor-core kernels take, layers that read another layer's latents, layers without a feed-forward, sizes off every grid of 8.
The weights are drawn here (not by the package), with queries scaled so that attention is peaked, every value representable
in bfloat16.
"""
from __future__ import annotations

import math

import torch

from potipel_tiny import make_engine  # noqa: F401  (an engine over given weights; nothing in it is one design's)


def lightning(heads, dim, vdim, decay):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def yarn(factor, original, fast=32.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=1e4, scaling=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": base}}
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def moe(ff, experts, top, count, keep):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def config(width, vocab, alpha, layers, eps=1e-5):
    return {"architecture": "Nidorax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": layers}


_Y = yarn(8.0, 256)
# A: both mixers, latents borrowed twice, a layer without a feed-forward, a second layer with latents of its own
CONFIG_A = config(72, 210, 1.5, [
    layer(lightning(3, 16, 24, [0.4, 0.9, 0.995]), moe(24, 6, 2, 3, 2)),
    layer(latent(3, 16, 8, 12, 24, 0.3, 5e4, _Y), moe(20, 8, 3, 2, 1)),
    layer(latent(5, 12, 8, 20, 24, 0.25, 5e4, _Y, kv_from=1), None),
    layer(latent(2, 24, 4, 16, 40, 0.2, 1e4, yarn(4.0, 64, 16.0, 2.0)), moe(24, 6, 1, 1, 1)),
    layer(latent(1, 8, 8, 8, 24, 0.35, 5e4, _Y, kv_from=1), moe(16, 4, 2, 4, 3)),
], eps=1e-5)
# B: sizes the tensor-core kernels take (cached rows of 128 and 64)
CONFIG_B = config(128, 340, 2.5, [
    layer(latent(8, 64, 32, 64, 96, 0.1, 1e5, yarn(16.0, 128)), moe(64, 8, 2, 4, 2)),
    layer(lightning(4, 64, 128, [0.7, 0.97, 0.99, 0.999]), moe(72, 16, 4, 8, 3)),
    layer(latent(4, 128, 32, 128, 96, 0.08, 1e5, yarn(16.0, 128), kv_from=0), moe(64, 4, 2, 2, 2)),
    layer(latent(4, 32, 16, 64, 48, 0.15, 2e4, None), None),
    layer(lightning(2, 128, 64, [0.95, 0.9995]), moe(64, 8, 1, 2, 1)),
], eps=1e-6)
# C: nothing on a grid of 8; one expert chosen; groups of one; one turning pair
CONFIG_C = config(100, 97, 1.6, [
    layer(latent(3, 10, 6, 14, 22, 0.35, 300.0, yarn(2.0, 40, 8.0, 1.5)), moe(14, 5, 1, 5, 2)),
    layer(lightning(3, 10, 6, [0.6, 0.98, 0.99]), moe(22, 6, 2, 2, 1)),
    layer(latent(2, 9, 2, 7, 11, 0.4, 50.0, None), moe(10, 3, 1, 3, 1)),
    layer(latent(7, 5, 6, 3, 22, 0.4, 300.0, yarn(2.0, 40, 8.0, 1.5), kv_from=0), None),
], eps=3e-6)
# D: a latent attention alone, without a feed-forward: what it does shows in the logits undiluted
CONFIG_D = config(64, 120, 0.5, [layer(latent(2, 32, 12, 16, 40, 0.2, 1e4, yarn(32.0, 100)), None)])
# E: recurrences only (no cache at all): decays of zero and one; every expert chosen
CONFIG_E = config(56, 130, 1.0, [layer(lightning(3, 32, 8, [0.0, 1.0, 0.9]), moe(16, 4, 4, 2, 2)),
                                 layer(lightning(7, 8, 16, [0.5, 0.8, 0.9, 0.95, 0.99, 0.999, 0.9999]), None)])
# F: a cached row wider than the tensor-core kernels take; every expert chosen, so that no choice can fall otherwise
CONFIG_F = config(96, 150, 3.0, [
    layer(latent(2, 40, 24, 32, 136, 0.15, 1e6, yarn(40.0, 4096, 64.0, 0.5)), moe(32, 6, 6, 1, 1)),
    layer(lightning(2, 48, 40, [0.99, 0.9]), moe(24, 3, 3, 3, 3)),
    layer(latent(6, 20, 24, 24, 136, 0.2, 1e6, yarn(40.0, 4096, 64.0, 0.5), kv_from=0), moe(16, 4, 4, 4, 4)),
], eps=1e-3)
# G: tensor-core sizes with every expert chosen
CONFIG_G = config(192, 200, 2.0 ** 0.5, [
    layer(lightning(6, 32, 32, [0.3, 0.8, 0.95, 0.99, 0.995, 0.9999]), moe(80, 3, 3, 1, 1)),
    layer(latent(6, 32, 64, 32, 64, 0.12, 1e4, yarn(4.0, 300)), moe(64, 2, 2, 2, 2)),
    layer(lightning(1, 256, 32, [0.97]), None),
], eps=1e-6)

CONFIGS = {"A": (CONFIG_A, 16), "B": (CONFIG_B, 16), "C": (CONFIG_C, 8), "D": (CONFIG_D, 32), "E": (CONFIG_E, 16),
           "F": (CONFIG_F, 16), "G": (CONFIG_G, 16)}   # name -> (config, page size)


def make_weights(cfg: dict, seed: int, peak: float = 1.5, decided: bool = False) -> dict:
    """Seeded weights by tensor name.  peak: the standard deviation the attention scores are scaled to.  decided: the routers'
    corrections lie further apart than any two scores can, so that no rounding moves a choice (the weights still depend on
    the token)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    rnd = lambda *shape, std=1.0, mean=0.0: (mean + torch.randn(tuple(shape), generator=g) * std).to(torch.bfloat16).float()
    gain = lambda *shape: rnd(*shape, std=0.1, mean=1.0)
    w = {"embed": rnd(cfg["vocab"], W), "final.norm": rnd(W, std=0.1)}
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}", lay["mixer"]
        for q in (1, 2) if lay["mlp"] is not None else (1,):
            w[f"{p}.norm{q}"] = rnd(W, std=0.15)           # stored around zero
        x = p + ".mix."
        if lay["type"] == "lightning":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            w[x + "q"] = rnd(H * D, W, std=1.5 / math.sqrt(W))
            w[x + "k"] = rnd(H * D, W, std=1.5 / math.sqrt(W))
            w[x + "v"] = rnd(H * V, W, std=1.5 / math.sqrt(W))
            w[x + "g"] = rnd(H * V, W, std=1.5 / math.sqrt(W))
            w[x + "norm"] = gain(H * V)
            w[x + "o"] = rnd(W, H * V, std=2.0 / math.sqrt(H * V))
        else:
            H, D, R, V, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w[x + "q"] = rnd(H * (D + R), W, std=peak / (m["scale"] * math.sqrt(D + R)) / math.sqrt(W))
            if m.get("kv_from") is None:
                w[x + "dkv"] = rnd(C + R, W, std=1.0 / math.sqrt(W))
                w[x + "dkv.norm"] = gain(C)
            w[x + "uk"] = rnd(H * D, C, std=1.0 / math.sqrt(C))
            w[x + "uv"] = rnd(H * V, C, std=1.5 / math.sqrt(C))
            w[x + "o"] = rnd(W, H * V, std=1.5 / math.sqrt(H * V))
        ff = lay["mlp"]
        if ff is None:
            continue
        y, F, E = p + ".mlp.", ff["expert"]["ff"], ff["router"]["experts"]
        for e in range(E):
            w[f"{y}e{e}.up"] = rnd(F, W, std=1.2 / math.sqrt(W))
            w[f"{y}e{e}.down"] = rnd(W, F, std=1.2 / math.sqrt(F))
        w[y + "router"] = rnd(E, W, std=2.0 / math.sqrt(W))
        w[y + "correction"] = rnd(E, std=0.2, mean=-0.3)          # changes choices and makes many choice scores negative
        if decided:
            w[y + "correction"] = (torch.randperm(E, generator=g).float() - E / 2) * 1.25
    return w


def random_config(seed: int, large: bool = False) -> dict:
    """Sizes, constants and layer order drawn from a seed.  large: sizes of some hundreds with heads of 32 to 128."""
    import random
    rng = random.Random(seed)
    pick = rng.choice
    width = pick([192, 320, 384, 512]) if large else pick([40, 56, 72, 88, 100, 128, 136])
    dims = [32, 64, 128] if large else [4, 8, 10, 16, 24, 32, 48, 64]
    ranks = [32, 64, 96, 112, 256] if large else [5, 12, 16, 30, 48, 64, 100]
    layers, own = [], []
    for n in range(rng.randint(2, 5)):
        r = rng.random()
        if r < 0.45:
            heads = rng.randint(1, 6)
            layers.append(lightning(heads, pick(dims), pick(dims), [pick([0.0, 0.3, 0.9, 0.99, 0.999, 1.0, rng.random()]) for _ in range(heads)]))
        elif r < 0.8 or not own:
            rot = pick([16, 32, 64]) if large else pick([2, 4, 6, 8, 16])
            scaling = None if rng.random() < 0.2 else yarn(pick([1.0, 2.0, 7.5, 40.0]), pick([32, 100, 4096]), pick([4.0, 32.0]), pick([0.5, 1.0, 2.0]))
            own.append(n)
            layers.append(latent(rng.randint(1, 6), pick(dims), rot, pick(dims), pick(ranks), rng.uniform(0.05, 0.5), pick([50.0, 1e4, 1e6]), scaling))
        else:
            src = pick(own)
            m = layers[src]["mixer"]
            layers.append(latent(rng.randint(1, 6), pick(dims), m["rot_dim"], pick(dims), m["kv_rank"], rng.uniform(0.05, 0.5), m["rot"]["base"],
                                 m["rot"].get("scaling"), kv_from=src))
        mlp = None
        if rng.random() < 0.75:
            count, per = pick([1, 2, 3, 4]), rng.randint(1, 3)
            keep = rng.randint(1, count)
            mlp = moe(pick([64, 80, 128]) if large else pick([8, 12, 20, 33]), count * per, rng.randint(1, keep * per), count, keep)
        layers[-1] = layer(layers[-1], mlp)
    return config(width, pick([61, 128, 200, 333]), pick([0.5, 1.0, 1.7, 4.0]), layers, eps=pick([1e-6, 1e-5, 1e-3]))
