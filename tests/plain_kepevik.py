"""A plain, slow implementation of the Kepevik design, one function per mechanism, whole sequences only.

Everything is written from the design's equations in torch on the CPU, in the dtype of the weights it is
given (the tests use float64), token by token where the design has a recurrence.  It shares no code with
the package: no kernels, no parts, no cache.  `forward(config, weights, tokens)` returns the logits at
every position of one sequence and, on request, the residual stream after every layer.

Notation: T tokens, W the model width, h the rows a sublayer reads, H heads, G key/value heads,
D the key size, V the value size.
"""
from __future__ import annotations

import torch


# ---- small pieces ------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    """An RMS norm whose stored weight is the gain's distance from one."""
    return rms_unit(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def gelu(x):
    return 0.5 * x * (1.0 + torch.erf(x / 2.0 ** 0.5))


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def log_sigmoid(x):
    return -softplus(-x)


def causal_conv(x, w):
    """y_t = sum_j w[:, j] x_(t - taps + 1 + j) per channel, zeros before the start.  x [T, C], w [C, taps]."""
    T, C = x.shape
    taps = w.shape[1]
    padded = torch.cat([x.new_zeros(taps - 1, C), x], dim=0)
    y = x.new_zeros(T, C)
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


def kv_head_of(h, heads, kv_heads):
    return h // (heads // kv_heads)


def sub(p, prefix):
    return {k[len(prefix) + 1:]: v for k, v in p.items() if k.startswith(prefix + ".")}


# ---- a matrix memory with exponential gates ------------------------------------------------------------------
def mlstm_gates(h, p, cap):
    """(log input gate, log forget gate), [T, H] each, both through a soft cap."""
    i = cap * torch.tanh((h @ p["i"].T + p["i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ p["f"].T + p["f.b"]) / cap))
    return i, f


def mlstm_scan(q, k, v, i, f):
    """The memory S and its normaliser n token by token, both scaled by exp(-m) for the running maximum m, which starts at 0.
    q, k [T, H, D], v [T, H, V], i, f [T, H]."""
    T, H, D = q.shape
    S, n, m = q.new_zeros(H, D, v.shape[-1]), q.new_zeros(H, D), q.new_zeros(H)
    out = q.new_zeros(T, H, v.shape[-1])
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        n = keep[:, None] * n + write[:, None] * k[t]
        m = m_new
        denom = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hdv,hd->hv", S, q[t]) / denom.unsqueeze(-1)
    return out


def mlstm(h, p, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ p["q"].T).view(T, H, D) * D ** -0.5
    k = (h @ p["k"].T).view(T, H, D)
    v = (h @ p["v"].T).view(T, H, V)
    i, f = mlstm_gates(h, p, m["gate_cap"])
    o = rms_unit(mlstm_scan(q, k, v, i, f), eps).reshape(T, H * V)
    return (o * p["norm"] * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


# ---- attention whose values are its keys before rotation --------------------------------------------------------
def rotate_halves(x, dims, base):
    """x [T, heads, D]: the first dims channels turn, channel i against channel i + dims/2, by position * base^(-2i/dims)."""
    T, half = x.shape[0], dims // 2
    f = torch.tensor(base, dtype=x.dtype) ** (-2.0 * torch.arange(half, dtype=x.dtype) / max(dims, 1))
    a = torch.arange(T, dtype=x.dtype).unsqueeze(1) * f
    c, s = torch.cos(a).unsqueeze(1), torch.sin(a).unsqueeze(1)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def keys_as_values_attention(h, p, m):
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ p["q"].T).view(T, H, D)
    v = (h @ p["k"].T).view(T, G, D)
    q, k = rotate_halves(q, m["rot"]["dims"], m["rot"]["base"]), rotate_halves(v, m["rot"]["dims"], m["rot"]["base"])
    visible = torch.tril(torch.ones(T, T, dtype=torch.bool))
    heads = []
    for hh in range(H):
        g = kv_head_of(hh, H, G)
        s = ((q[:, hh] @ k[:, g].T) * m["scale"]).masked_fill(~visible, float("-inf"))
        heads.append(torch.softmax(s, dim=-1) @ v[:, g])
    return torch.cat(heads, dim=-1) @ p["o"].T


# ---- delta rule with a decay per key channel ----------------------------------------------------------------------
def channel_decay(h, p, H, D):
    """[T, H, D]: exp(-exp(A_log_h) softplus(a2 (a1 h) + dt_bias))."""
    z = (h @ p["a1"].T) @ p["a2"].T + p["dt_bias"]
    return torch.exp(-torch.exp(p["A_log"]).view(1, H, 1) * softplus(z).view(-1, H, D))


def delta_scan(q, k, v, beta, decay):
    """q, k [T, H, D] (each head's), v [T, H, V], beta [T, H], decay [T, H, D]: decay the rows, correct, write, read."""
    T, H, D = q.shape
    S = q.new_zeros(H, D, v.shape[-1])
    out = q.new_zeros(T, H, v.shape[-1])
    for t in range(T):
        S = decay[t].unsqueeze(-1) * S
        u = beta[t].unsqueeze(-1) * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t].unsqueeze(-1) * u.unsqueeze(1)
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def channel_delta(h, p, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(silu(causal_conv(h @ p["q"].T, p["q.conv"])).view(T, G, D)) * D ** -0.5
    k = unit(silu(causal_conv(h @ p["k"].T, p["k.conv"])).view(T, G, D))
    v = silu(causal_conv(h @ p["v"].T, p["v.conv"])).view(T, H, V)
    of = torch.tensor([kv_head_of(hh, H, G) for hh in range(H)])
    o = delta_scan(q[:, of], k[:, of], v, torch.sigmoid(h @ p["b"].T), channel_decay(h, p, H, D))
    o = rms_unit(o, eps) * p["norm"] * torch.sigmoid((h @ p["g1"].T) @ p["g2"].T).view(T, H, V)
    return o.reshape(T, H * V) @ p["o"].T


def parallel(h, p, m, eps):
    return (m["left_scale"] * keys_as_values_attention(h, sub(p, "left"), m["left"])
            + m["right_scale"] * channel_delta(h, sub(p, "right"), m["right"], eps))


# ---- feed-forward -----------------------------------------------------------------------------------------
def dense_ff(h, p):
    return gelu(h @ p["up"].T + p["up.b"]) @ p["down"].T + p["down.b"]


def gated_ff(h, p):
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def route(h, p, r):
    """(chosen experts [T, top], their weights [T, top], margin [T]): the softmax over every output, a correction for the
    choice only, weights not renormalised.  margin: the last chosen choice score minus the best one left out."""
    top, n = r["top"], r["experts"] + r.get("identity", 0)
    s = torch.softmax(h @ p["router"].T, dim=-1)
    order = (s + p["correction"]).sort(dim=-1, descending=True)
    ids = order.indices[:, :top]
    margin = (order.values[:, top - 1] - order.values[:, top]) if top < n else torch.full((h.shape[0],), float("inf"), dtype=h.dtype)
    return ids, s.gather(1, ids), margin


def moe_ff(h, p, mlp):
    """Experts from `experts` on are the input itself; a shared expert runs for every token behind a gate of one number."""
    r = mlp["router"]
    ids, wts, _ = route(h, p, r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(ids.shape[1]):
            e = int(ids[t, j])
            y = gated_ff(h[t:t + 1], sub(p, f"e{e}"))[0] if e < r["experts"] else h[t]
            out[t] = out[t] + wts[t, j] * y
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ p["shared.sg"].T) * gated_ff(h, sub(p, "shared"))
    return out


# ---- the model --------------------------------------------------------------------------------------------
def forward(config, weights, tokens, want_layers=False, margins=None):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer).  margins: a list that
    receives every routed layer's routing margins [T]."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    after = []
    for i, layer in enumerate(config["layers"]):
        p = sub(weights, f"l{i}")
        mixer = {"mlstm": mlstm, "parallel": parallel}[layer["type"]]
        y = mixer(norm_around_zero(x, p["norm1"], eps), sub(p, "mix"), layer["mixer"], eps)
        x = x + norm_around_zero(y, p["norm1b"], eps) * p["ls1"]
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm_around_zero(x, p["norm2"], eps)
            if mlp["kind"] == "dense":
                y = dense_ff(h, sub(p, "mlp"))
            else:
                if margins is not None:
                    margins.append(route(h, sub(p, "mlp"), mlp["router"])[2])
                y = moe_ff(h, sub(p, "mlp"), mlp)
            x = x + norm_around_zero(y, p["norm2b"], eps) * p["ls2"]
        after.append(x)
    logits = norm_around_zero(x, weights["final.norm"], eps) @ weights["embed"].T
    return (logits, torch.stack(after)) if want_layers else logits
