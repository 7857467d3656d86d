"""Tiny Kepevik configurations and weights for the tests.

The configurations differ from each other in every size and constant and include the corner values: convolutions of one tap
(none at all) and of many, one head, as many kv heads as query heads and fewer, key and value sizes that differ and value sizes
above and off a block of 64 columns, rotations of no, some and all channels, gate caps that hardly bend and that bend everything,
one expert chosen and all of them, no identity experts and many, no shared expert, layers without a feed-forward, sizes off every
grid of 8.  The weights are drawn here (not by the package), with queries scaled so that attention is peaked, gates and decays
spread between fast and slow, every value representable in bfloat16.
"""
from __future__ import annotations

import math

import torch


def mlstm(heads, dim, vdim, gate_cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def parallel(heads, kv_heads, dim, scale, rot_dims, rot_base, r_heads, r_kv, r_dim, r_vdim, r_conv, left_scale=0.7, right_scale=0.9):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                 "rot": {"dims": rot_dims, "base": rot_base}},
        "right": {"heads": r_heads, "kv_heads": r_kv, "dim": r_dim, "vdim": r_vdim, "conv": r_conv},
        "left_scale": left_scale, "right_scale": right_scale}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, identity, top, shared):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def config(width, vocab, scale, layers, eps=1e-5):
    return {"architecture": "Kepevik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


# A: both mixers and both feed-forwards; rotation of a part of the head
CONFIG_A = config(64, 200, 2.0, [
    layer(mlstm(2, 16, 24, 6.0), dense(40)),
    layer(parallel(4, 2, 16, 0.3, 8, 10000.0, r_heads=4, r_kv=2, r_dim=16, r_vdim=8, r_conv=3), moe(24, 6, 2, 2, 32)),
    layer(mlstm(1, 8, 16, 20.0), moe(16, 4, 1, 1, 24)),
])
# B: sizes the tensor-core kernels take; fewer kv heads than heads everywhere; value sizes above a block of 64 columns
CONFIG_B = config(128, 333, 5.0, [
    layer(parallel(8, 2, 64, 0.125, 64, 100000.0, r_heads=4, r_kv=1, r_dim=64, r_vdim=32, r_conv=4, left_scale=1.3, right_scale=0.6),
          dense(64)),
    layer(mlstm(4, 32, 72, 15.0), moe(64, 8, 3, 3, 48)),
    layer(parallel(2, 2, 128, 0.1, 32, 5000.0, r_heads=2, r_kv=2, r_dim=128, r_vdim=64, r_conv=2), None),
    layer(mlstm(2, 64, 128, 9.0), dense(136)),
], eps=1e-6)
# C: nothing on a grid of 8; a convolution of one tap; one expert chosen; no identity experts, no shared expert
CONFIG_C = config(100, 97, 1.0, [
    layer(parallel(3, 3, 10, 0.35, 6, 100.0, r_heads=3, r_kv=3, r_dim=12, r_vdim=10, r_conv=1), moe(14, 5, 0, 1, 0)),
    layer(mlstm(3, 10, 6, 2.0), dense(22)),
    layer(mlstm(5, 7, 67, 11.0), moe(10, 3, 4, 2, 0)),
], eps=3e-6)
# D: the matrix memory alone, without a feed-forward
CONFIG_D = config(64, 120, 3.0, [layer(mlstm(2, 48, 40, 10.0), None)])
# E: attention beside the delta rule, alone, no rotation
CONFIG_E = config(48, 150, 2.0, [layer(parallel(2, 1, 24, 0.2, 0, 10000.0, r_heads=2, r_kv=1, r_dim=20, r_vdim=12, r_conv=5), None)])
# F: recurrences, long memories; every expert chosen, the identity experts among them
CONFIG_F = config(56, 130, 0.5, [
    layer(mlstm(7, 8, 8, 30.0), moe(16, 2, 2, 4, 8)), layer(mlstm(2, 24, 130, 4.0), None),
    layer(parallel(1, 1, 40, 0.15, 40, 1e6, r_heads=6, r_kv=2, r_dim=24, r_vdim=36, r_conv=2, left_scale=0.4, right_scale=1.5), dense(24))])
# G: large heads of the recurrences
CONFIG_G = config(72, 90, 4.0, [
    layer(mlstm(1, 256, 24, 7.0), None),
    layer(parallel(6, 3, 8, 0.5, 2, 50.0, r_heads=1, r_kv=1, r_dim=200, r_vdim=36, r_conv=6), moe(12, 7, 1, 5, 20))])

CONFIGS = {"A": (CONFIG_A, 16), "B": (CONFIG_B, 16), "C": (CONFIG_C, 8), "D": (CONFIG_D, 16), "E": (CONFIG_E, 32),
           "F": (CONFIG_F, 16), "G": (CONFIG_G, 16)}   # name -> (config, page size)


def make_weights(cfg: dict, seed: int, peak: float = 1.5, slow: float = 0.0, rank: int = 0) -> dict:
    """Seeded weights by tensor name.  peak: the standard deviation the attention scores are scaled to; slow: shifts the
    recurrences' decays toward one (larger: longer memory); rank: of the low-rank projections (0: drawn, on and off a grid)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    rnd = lambda *shape, std=1.0, mean=0.0: (mean + torch.randn(tuple(shape), generator=g) * std).to(torch.bfloat16).float()
    gain = lambda *shape: rnd(*shape, std=0.1, mean=1.0)
    w = {"embed": rnd(cfg["vocab"], W, std=1.0 / cfg["embedding"]["scale"]), "final.norm": rnd(W, std=0.1)}
    for i, lay in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}", lay["mixer"], lay["type"]
        for q in (1, 2) if lay["mlp"] is not None else (1,):
            w[f"{p}.norm{q}"], w[f"{p}.norm{q}b"] = rnd(W, std=0.1), rnd(W, std=0.1)
            w[f"{p}.ls{q}"] = rnd(W, std=0.3, mean=0.8)
        x = p + ".mix."
        if kind == "mlstm":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            w[x + "q"] = rnd(H * D, W, std=1.5 / math.sqrt(W))
            w[x + "k"] = rnd(H * D, W, std=1.0 / math.sqrt(W))
            w[x + "v"] = rnd(H * V, W, std=1.0 / math.sqrt(W))
            w[x + "g"] = rnd(H * V, W, std=1.5 / math.sqrt(W))
            w[x + "i"] = rnd(H, W, std=2.5 / math.sqrt(W))
            w[x + "i.b"] = rnd(H, std=1.5, mean=-0.5)
            w[x + "f"] = rnd(H, W, std=1.5 / math.sqrt(W))
            w[x + "f.b"] = rnd(H, std=1.0, mean=2.0 + slow)
            w[x + "norm"] = gain(H * V)
            w[x + "o"] = rnd(W, H * V, std=1.0 / math.sqrt(H * V))
        else:
            a, b = m["left"], m["right"]
            H, G, D = a["heads"], a["kv_heads"], a["dim"]
            y = x + "left."
            w[y + "q"] = rnd(H * D, W, std=peak / (a["scale"] * math.sqrt(D)) / math.sqrt(W))
            w[y + "k"] = rnd(G * D, W, std=1.0 / math.sqrt(W))
            w[y + "o"] = rnd(W, H * D, std=1.0 / math.sqrt(H * D))
            H, G, D, V, taps = b["heads"], b["kv_heads"], b["dim"], b["vdim"], b["conv"]
            y = x + "right."
            for n, c in (("q", G * D), ("k", G * D), ("v", H * V)):
                w[y + n] = rnd(c, W, std=1.5 / math.sqrt(W))
                conv = rnd(c, taps, std=0.3)
                conv[:, -1] += 1.0          # the current token's tap carries most of the weight
                w[y + n + ".conv"] = conv.to(torch.bfloat16).float()
            w[y + "b"] = rnd(H, W, std=1.5 / math.sqrt(W))
            ra, rg = (rank, rank) if rank else (int(torch.randint(1, 20, (1,), generator=g)), int(torch.randint(1, 4, (1,), generator=g)) * 8)
            w[y + "a1"] = rnd(ra, W, std=1.0 / math.sqrt(W))
            w[y + "a2"] = rnd(H * D, ra, std=1.0 / math.sqrt(ra))
            w[y + "A_log"] = rnd(H, std=0.7, mean=-slow)
            w[y + "dt_bias"] = rnd(H * D, std=1.5, mean=-1.0 - slow)
            w[y + "g1"] = rnd(rg, W, std=1.5 / math.sqrt(W))
            w[y + "g2"] = rnd(H * V, rg, std=1.0 / math.sqrt(rg))
            w[y + "norm"] = gain(V)
            w[y + "o"] = rnd(W, H * V, std=1.0 / math.sqrt(H * V))
        ff = lay["mlp"]
        if ff is None:
            continue
        y = p + ".mlp."
        if ff["kind"] == "dense":
            F = ff["ff"]
            w[y + "up"], w[y + "up.b"] = rnd(F, W, std=1.5 / math.sqrt(W)), rnd(F, std=0.5)
            w[y + "down"], w[y + "down.b"] = rnd(W, F, std=1.0 / math.sqrt(F)), rnd(W, std=0.5)
            continue

        def gated(at, F):
            w[at + "gate"] = rnd(F, W, std=1.5 / math.sqrt(W))
            w[at + "up"] = rnd(F, W, std=1.0 / math.sqrt(W))
            w[at + "down"] = rnd(W, F, std=1.5 / math.sqrt(F))
        for e in range(ff["router"]["experts"]):
            gated(f"{y}e{e}.", ff["expert"]["ff"])
        n = ff["router"]["experts"] + ff["router"].get("identity", 0)
        w[y + "router"] = rnd(n, W, std=2.0 / math.sqrt(W))
        w[y + "correction"] = rnd(n, std=0.3)          # large enough to change choices and to make choice scores negative
        if ff.get("shared") is not None:
            gated(y + "shared.", ff["shared"]["ff"])
            w[y + "shared.sg"] = rnd(1, W, std=1.5 / math.sqrt(W))
    return w


def random_config(seed: int, large: bool = False) -> dict:
    """Sizes, constants and layer order drawn from a seed.  large: sizes of some hundreds with heads of 32 to 128."""
    import random
    rng = random.Random(seed)
    pick = rng.choice
    width = pick([192, 256, 320, 384]) if large else pick([40, 56, 72, 88, 100, 128, 136])
    dims = [32, 64, 128] if large else [4, 8, 10, 16, 24, 32, 48, 64]
    vdims = [32, 64, 128, 192] if large else [4, 7, 8, 12, 16, 20, 32, 64, 70]
    layers = []
    for n in range(rng.randint(2, 5)):
        if rng.random() < 0.5:
            mixer = mlstm(rng.randint(1, 6), pick(dims), pick(vdims), pick([1.0, 5.0, 15.0, 40.0]))
        else:
            kv, r_kv, dim = pick([1, 2, 4]), pick([1, 2, 3]), pick(dims)
            mixer = parallel(kv * rng.randint(1, 3), kv, dim, rng.uniform(0.05, 0.5), rng.randint(0, dim // 2) * 2, pick([10.0, 1e4, 1e6]),
                             r_heads=r_kv * rng.randint(1, 2), r_kv=r_kv, r_dim=pick(dims), r_vdim=pick(vdims), r_conv=rng.randint(1, 6),
                             left_scale=rng.uniform(0.3, 1.5), right_scale=rng.uniform(0.3, 1.5))
        r = rng.random()
        if r < 0.2:
            mlp = None
        elif r < 0.5:
            mlp = dense(pick([256, 344]) if large else pick([8, 12, 24, 40]))
        else:
            experts, identity = rng.randint(1, 9), rng.randint(0, 3)
            mlp = moe(pick([64, 80]) if large else pick([8, 12, 20]), experts, identity, rng.randint(1, min(4, experts + identity)),
                      pick([0, 40, 64]) if large else pick([0, 6, 16]))
        layers.append(layer(mixer, mlp))
    return config(width, pick([61, 128, 200, 333]), pick([0.5, 1.0, 4.0, 16.0]), layers, eps=pick([1e-6, 1e-5, 1e-3]))


def make_engine(cfg, weights, dtype, page, num_blocks, max_tokens=512, max_seqs=4, poison=True, graphs=False, max_seq_len=None):
    from llm_b200.config import EngineOptions
    from llm_b200.engine.engine import Engine
    opts = EngineOptions(dtype=dtype, kv_block_size=page, max_num_seqs=max_seqs, max_num_batched_tokens=max_tokens,
                         num_kv_blocks=num_blocks, use_cuda_graphs=graphs, poison_freed_pages=poison,
                         max_seq_len=max_seq_len or min(num_blocks * page, 4096))
    return Engine(None, opts, random_config=cfg, tensors={k: v.clone() for k, v in weights.items()})
