"""A plain, slow implementation of the Nidorax design, one function per mechanism, whole sequences only.

Everything is written from the design's equations in torch on the CPU, in the dtype of the weights it is
given (the tests use float64), token by token where the design has a recurrence.  It shares no code with
the package: no kernels, no parts, no cache.  `forward(config, weights, tokens)` returns the logits at
every position of one sequence and, on request, the residual stream after every layer.

Notation: T tokens, W the model width, x the residual rows a sublayer reads, H heads, D the unrotated
query/key size, R the rotated size, V the value size, C the latent size.
"""
from __future__ import annotations

import math

import torch


# ---- small pieces ------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def centred_norm(x, w, eps):
    """The model's norm: its weight is stored as the distance from one."""
    return rms_unit(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def relu_squared(x):
    return torch.relu(x) ** 2


def sub(p, prefix):
    return {k[len(prefix) + 1:]: v for k, v in p.items() if k.startswith(prefix + ".")}


# ---- rotation ----------------------------------------------------------------------------------------------
def yarn(dims, base, scaling=None):
    """(frequencies [dims / 2], factor on cos and sin).  Frequencies that turn often within the original length keep
    their value, those that turn seldom are divided by `factor`, a linear ramp over the index in between."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    def index_of(turns):      # the (fractional) pair whose frequency makes `turns` turns within the original length
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index_of(scaling["fast"])), 0)
    hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_halves(x, positions, freqs, amp, ang=None):
    """x [..., T, dims]: channel i turns against channel i + dims / 2 by position * f_i (or by given angles [T, dims / 2]);
    cos and sin carry `amp`."""
    half = len(freqs)
    if ang is None:
        ang = positions.to(x.dtype).unsqueeze(-1) * torch.tensor(freqs, dtype=x.dtype)
    c, s = torch.cos(ang) * amp, torch.sin(ang) * amp
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


# ---- latent attention --------------------------------------------------------------------------------------
def latents(x, p, m, eps):
    """What a layer with a down-projection keeps per token: (latent [T, C], turned key part [T, R])."""
    T, C = x.shape[0], m["kv_rank"]
    down = x @ p["dkv"].T
    c = rms_norm(down[:, :C], p["dkv.norm"], eps)
    freqs, amp = yarn(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    return c, rotate_halves(down[:, C:], torch.arange(T), freqs, amp)


def latent_attention(x, p, m, kept):
    """Causal softmax attention; `kept` is what latents() of this layer, or of the layer it borrows from, returned."""
    T = x.shape[0]
    H, D, R, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, turned = kept
    q = (x @ p["q"].T).view(T, H, D + R)
    freqs, amp = yarn(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    k = (c @ p["uk"].T).view(T, H, D)
    v = (c @ p["uv"].T).view(T, H, V)
    hidden = torch.ones(T, T, dtype=torch.bool).triu(1)
    heads = []
    for h in range(H):
        qr = rotate_halves(q[:, h, D:], torch.arange(T), freqs, amp)
        s = (q[:, h, :D] @ k[:, h].T + qr @ turned.T) * m["scale"]
        heads.append(torch.softmax(s.masked_fill(hidden, float("-inf")), dim=-1) @ v[:, h])
    return torch.cat(heads, dim=-1) @ p["o"].T


# ---- lightning attention -----------------------------------------------------------------------------------
def lightning_recurrence(q, k, v, decay, S=None):
    """S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head.  q, k [T, H, D], v [T, H, V] -> ([T, H, V], S)."""
    T, H, D = q.shape
    d = torch.tensor(decay, dtype=q.dtype).view(H, 1, 1)
    S = q.new_zeros(H, D, v.shape[2]) if S is None else S
    out = q.new_zeros(T, H, v.shape[2])
    for t in range(T):
        S = d * S + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def lightning(x, p, m, eps):
    """The recurrence on silu projections, one RMS norm over all heads together, a sigmoid gate, the output projection."""
    T = x.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = silu(x @ p["q"].T).view(T, H, D)
    k = silu(x @ p["k"].T).view(T, H, D)
    v = silu(x @ p["v"].T).view(T, H, V)
    o, _ = lightning_recurrence(q, k, v, m["decay"])
    o = rms_norm(o.reshape(T, H * V), p["norm"], eps) * torch.sigmoid(x @ p["g"].T)
    return o @ p["o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------
def route(x, p, r):
    """(chosen experts [T, top], their weights [T, top], margin [T]): softmax scores over all experts, a correction for the
    choice only, experts outside the best groups (by their largest choice score) shut out, the chosen scores divided by
    their sum.  margin: how far the nearest other choice (of an expert or of a group) was, inf where there is none."""
    E, top = r["experts"], r["top"]
    count, keep = r["groups"]["count"], r["groups"]["keep"]
    s = torch.softmax(x @ p["router"].T, dim=-1)
    choice = s + p["correction"]
    T, per = x.shape[0], E // count
    inf = float("inf")
    margin = torch.full((T,), inf, dtype=x.dtype)
    ids = torch.zeros(T, top, dtype=torch.long)
    for t in range(T):
        best = [(float(choice[t, g * per:(g + 1) * per].max()), g) for g in range(count)]
        best.sort(key=lambda b: (-b[0], b[1]))
        kept = {g for _, g in best[:keep]}
        allowed = [(float(choice[t, e]), e) for e in range(E) if e // per in kept]
        allowed.sort(key=lambda b: (-b[0], b[1]))
        ids[t] = torch.tensor([e for _, e in allowed[:top]])
        if keep < count:
            margin[t] = best[keep - 1][0] - best[keep][0]
        if top < len(allowed):
            margin[t] = min(float(margin[t]), allowed[top - 1][0] - allowed[top][0])
    w = s.gather(1, ids)
    return ids, w / (w.sum(dim=-1, keepdim=True) + 1e-20), margin


def expert_ff(x, p):
    return relu_squared(x @ p["up"].T) @ p["down"].T


def moe_ff(x, p, mlp):
    ids, w, _ = route(x, p, mlp["router"])
    out = torch.zeros_like(x)
    for e in range(mlp["router"]["experts"]):
        rows, place = torch.nonzero(ids == e, as_tuple=True)
        if rows.numel():
            out[rows] += w[rows, place].unsqueeze(-1) * expert_ff(x[rows], sub(p, f"e{e}"))
    return out


# ---- the model ---------------------------------------------------------------------------------------------
def forward(config, weights, tokens, want_layers=False, margins=None):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer).  margins: a list that receives
    every routed layer's margins [T]."""
    eps, alpha = config["norm"]["eps"], config["postln_alpha"]
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kept, after = {}, []
    for i, layer in enumerate(config["layers"]):
        p, m = sub(weights, f"l{i}"), layer["mixer"]
        if layer["type"] == "lightning":
            y = lightning(x, sub(p, "mix"), m, eps)
        else:
            src = m.get("kv_from")
            if src is None:
                kept[i] = latents(x, sub(p, "mix"), m, eps)
            y = latent_attention(x, sub(p, "mix"), m, kept[i if src is None else src])
        x = centred_norm(alpha * x + y, p["norm1"], eps)
        if layer.get("mlp") is not None:
            if margins is not None:
                margins.append(route(x, sub(p, "mlp"), layer["mlp"]["router"])[2])
            x = centred_norm(alpha * x + moe_ff(x, sub(p, "mlp"), layer["mlp"]), p["norm2"], eps)
        after.append(x)
    logits = centred_norm(x, weights["final.norm"], eps) @ weights["embed"].T
    return (logits, torch.stack(after)) if want_layers else logits
