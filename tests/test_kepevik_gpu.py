"""GPU tests of the Kepevik design against the plain implementation (tests/plain_kepevik.py): each mechanism alone,
then whole models under every way of cutting the work."""
import json
import math
from types import SimpleNamespace

import pytest
import torch

import plain_kepevik as P
import replay
from kepevik_tiny import CONFIGS, config, layer, make_engine, make_weights, mlstm, parallel, random_config
from tiny import max_err, random_tokens

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 3e-5, "bfloat16": 5e-2}       # whole models, relative to the largest logit
KTOL = {"float32": 4e-6, "bfloat16": 6e-3}      # kernels alone: one rounding of the output


def dev(t, dtype="float32"):
    return t.to(device="cuda", dtype=DT[dtype]).contiguous()


def bf(t):
    return t.to(torch.bfloat16).float()


def i32(xs):
    return torch.tensor(xs, dtype=torch.int32, device="cuda")


def step_ctx(lens, slots):
    """What the kernels read of a step: entries of lens tokens laid end to end, each with its state slot."""
    cu, entry = [0], []
    for e, n in enumerate(lens):
        cu.append(cu[-1] + n)
        entry += [e] * n
    return SimpleNamespace(n_tokens=cu[-1], n_entries=len(lens), cu_tokens=i32(cu), token_entry=i32(entry), state_slots=i32(slots))


def split_steps(total, cuts):
    out, at, k = [], 0, 0
    while at < total:
        n = min(cuts[k % len(cuts)], total - at)
        out.append((at, at + n))
        at, k = at + n, k + 1
    return out


# ---- each mechanism alone ---------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hidden,rows", [(8, 3), (100, 5), (512, 33), (2048, 4), (4104, 3), (8200, 2)])
def test_rms_norms_on_both_sides_of_the_residual_sum(dtype, hidden, rows):
    """x += mult * rms(y + bias) * post; out = rms(x) * pre; either half alone; y also as unsummed partial results."""
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(hidden)
    x, y, bias = torch.randn(rows, hidden, generator=g), bf(torch.randn(rows, hidden, generator=g)), torch.randn(hidden, generator=g)
    post, pre, eps, mult = torch.randn(hidden, generator=g), torch.randn(hidden, generator=g), 1e-3, 0.8
    d = lambda t: t.double()
    with_bias = lambda b: dev(y, dtype) if b is None else ops.BiasedRows(dev(y, dtype), dev(b))
    for b in (None, bias):
        want = d(x) + mult * P.rms_unit(d(y) + (0 if b is None else d(b)), eps) * d(post)
        resid, out = dev(x), torch.empty(rows, hidden, device="cuda", dtype=DT[dtype])
        ops.add_rmsnorms(resid, with_bias(b), dev(post), mult, dev(pre), out, rows, eps)
        assert max_err(resid, want) < 1e-6 and max_err(out, P.rms_unit(want, eps) * d(pre)) < KTOL[dtype]
        resid = dev(x)
        ops.add_rmsnorms(resid, with_bias(b), dev(post), mult, None, None, rows, eps)
        assert max_err(resid, want) < 1e-6
    parts = torch.randn(3, rows, hidden, generator=g)
    resid = dev(x)
    ops.add_rmsnorms(resid, ops.PartialSum(dev(parts), 3, rows, hidden, DT[dtype]), dev(post), mult, dev(pre), out, rows, eps)
    assert max_err(resid, d(x) + mult * P.rms_unit(d(parts).sum(0), eps) * d(post)) < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hidden,rows", [(8, 3), (100, 5), (2048, 4), (4096, 2), (8200, 2)])
def test_norms_take_a_sublayers_last_sums(dtype, hidden, rows):
    """Two mixers' rows with their scales; a routed feed-forward's rows with identity experts and a gated shared expert, the norm's
    output written over the input those experts pass."""
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(hidden + 1)
    x, a, b = torch.randn(rows, hidden, generator=g), bf(torch.randn(rows, hidden, generator=g)), torch.randn(2, rows, hidden, generator=g)
    post, pre, eps = torch.randn(hidden, generator=g), torch.randn(hidden, generator=g), 1e-4
    part = ops.PartialSum(dev(b), 2, rows, hidden, DT[dtype])
    pair = 0.7 * a.double() - 1.3 * b.double().sum(0)
    want = x.double() + P.rms_unit(pair, eps) * post.double()
    resid, out = dev(x), torch.empty(rows, hidden, device="cuda", dtype=DT[dtype])
    ops.add_rmsnorms(resid, ops.ScaledPair(dev(a, dtype), part, 0.7, -1.3), dev(post), 1.0, dev(pre), out, rows, eps)
    assert max_err(resid, want) < 2e-6 and max_err(out, P.rms_unit(want, eps) * pre.double()) < KTOL[dtype]
    top, E = 3, 4
    y, w, h = torch.randn(6, hidden, generator=g), torch.rand(rows, top, generator=g), bf(torch.randn(rows, hidden, generator=g))
    ids = torch.randint(0, E + 2, (rows, top), generator=g)
    ids[0, 0], ids[-1, -1] = E, E + 1
    slots = torch.where(ids < E, ids, torch.full_like(ids, -1))
    gate = torch.rand(rows, generator=g)
    terms = torch.where((ids < E).unsqueeze(-1), y.double()[slots.clamp(min=0)], h.double().unsqueeze(1))
    routed = (w.double().unsqueeze(-1) * terms).sum(1)
    for shared, scale in ((None, 0.0), (part, 1.0)):
        want = x.double() + 0.5 * P.rms_unit(routed + scale * gate.double().unsqueeze(1) * b.double().sum(0), eps) * post.double()
        resid, hd = dev(x), dev(h, dtype)
        rows_of = ops.WeightedRows(dev(y), i32(slots.flatten().tolist()), dev(w), top, rows, shared=shared, shared_gate=dev(gate) if shared else None,
                                   ids=i32(ids.flatten().tolist()), first_identity=E, x=hd)
        ops.add_rmsnorms(resid, rows_of, dev(post), 0.5, dev(pre), hd, rows, eps)
        assert max_err(resid, want) < 2e-6 and max_err(hd, P.rms_unit(want, eps) * pre.double()) < KTOL[dtype]


@pytest.mark.parametrize("rows,ff,width", [(129, 72, 64), (300, 328, 128), (1000, 1000, 512)])
def test_bias_and_activation_in_the_products_epilogue(rows, ff, width):
    """Many rows in bfloat16: gelu(x W^T + b) is made in the epilogue of the product; widths off the tile's among them."""
    from llm_b200.parts.linear import linear_act
    g = torch.Generator().manual_seed(rows)
    x, w, b = bf(torch.randn(rows, width, generator=g)), bf(torch.randn(ff, width, generator=g) / math.sqrt(width)), torch.randn(ff, generator=g)
    out = torch.empty(rows, ff, device="cuda", dtype=torch.bfloat16)
    assert linear_act(dev(x, "bfloat16"), dev(w, "bfloat16"), out, rows, "gelu", bias=dev(b))
    assert max_err(out, P.gelu(x.double() @ w.double().T + b.double())) < KTOL["bfloat16"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_scale_is_part_of_the_posts_gain(dtype):
    from llm_b200.models.spec import PartSpec
    from llm_b200.parts.base import build_part
    part = build_part("norm", PartSpec("rmsnorm", {"size": 40, "eps": 1e-5, "weight_name": "n", "centred": True, "scale_name": "s"}, "x"),
                      DT[dtype], torch.device("cuda"))
    w = {n: torch.randn(40, device="cuda") for n in part.parameters()}
    part.bind(w)
    assert sorted(w) == ["x.n", "x.s"] and max_err(part.gain, (1.0 + w["x.n"].double()) * w["x.s"].double()) < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["gelu", "silu"])
@pytest.mark.parametrize("rows,cols", [(3, 8), (7, 100), (33, 328)])
def test_activation_behind_a_bias(dtype, kind, rows, cols):
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(cols)
    x, b = bf(torch.randn(rows, cols, generator=g)), torch.randn(cols, generator=g)
    out = torch.empty(rows, cols, device="cuda", dtype=DT[dtype])
    act = {"gelu": P.gelu, "silu": P.silu}[kind]
    ops.bias_act_rows(out, dev(x, dtype), dev(b), rows, kind)
    assert max_err(out, act(x.double() + b.double())) < KTOL[dtype]
    parts = torch.randn(2, rows, cols, generator=g)
    ops.bias_act_rows(out, ops.PartialSum(dev(parts), 2, rows, cols, DT[dtype]), dev(b), rows, kind)
    assert max_err(out, act(parts.double().sum(0) + b.double())) < KTOL[dtype]


@pytest.mark.parametrize("dtype,gate_dtype", [("float32", "float32"), ("bfloat16", "bfloat16"), ("bfloat16", "float32")])
@pytest.mark.parametrize("H,V", [(1, 4), (3, 10), (2, 64), (4, 136), (2, 300)])
@pytest.mark.parametrize("own", [False, True])
def test_head_norm_with_a_sigmoid_gate(dtype, gate_dtype, H, V, own):
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 100 + V)
    T, col, eps = 9, 5, 1e-5
    x, gate = torch.randn(T, H * V, generator=g), bf(torch.randn(T, col + H * V + 3, generator=g))
    w = torch.randn(H * V if own else V, generator=g)
    ref = P.rms_unit(x.double().view(T, H, V), eps) * (w.double().view(H, V) if own else w.double())
    ref = ref.reshape(T, H * V) * torch.sigmoid(gate[:, col:col + H * V].double())
    out = torch.empty(T, H * V, device="cuda", dtype=DT[dtype])
    ops.head_rmsnorm_sigmoid(out, dev(x), dev(w), dev(gate, gate_dtype), col, T, H, eps)
    assert max_err(out, ref) < KTOL[dtype]
    half = gate * 0.5
    parts = ops.PartialSum(dev(torch.stack([half, half])), 2, T, gate.shape[1], DT[gate_dtype])
    ops.head_rmsnorm_sigmoid(out, dev(x), dev(w), parts, col, T, H, eps)
    assert max_err(out, ref) < KTOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,I,top", [(6, 2, 2), (1, 0, 1), (3, 3, 6), (12, 1, 4), (37, 5, 3), (4, 8, 2)])
@pytest.mark.parametrize("gated", [False, True])
def test_router_over_experts_and_identities_with_a_shared_gate(dtype, E, I, top, gated):
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(E * 10 + top)
    T, W = 50, 24
    h = bf(torch.randn(T, W, generator=g))
    p = {"router": bf(torch.randn(E + I, W, generator=g) * 0.5), "correction": bf(torch.randn(E + I, generator=g) * 0.2 - 0.3)}
    sg = bf(torch.randn(1, W, generator=g))
    ids_ref, w_ref, margin = P.route(h.double(), {k: v.double() for k, v in p.items()}, {"experts": E, "identity": I, "top": top})
    w = torch.cat([p["router"], sg]) if gated else p["router"]
    logits = torch.empty(T, w.shape[0], device="cuda")
    ids, wts = torch.empty(T * top, dtype=torch.int32, device="cuda"), torch.empty(T * top, device="cuda")
    gate = torch.full((T,), float("nan"), device="cuda") if gated else None
    ops.moe_route(dev(h, dtype), dev(w, dtype), dev(p["correction"]), logits, ids, wts, T, top, groups=(1, 1), softmax=True, gate_out=gate)
    ids, wts = ids.view(T, top).cpu().long(), wts.view(T, top).cpu()
    clear = margin > 1e-4
    assert int(clear.sum()) > T // 2 and torch.equal(ids[clear], ids_ref[clear]) and max_err(wts[clear], w_ref[clear]) < 1e-5
    if gated:
        assert max_err(gate, torch.sigmoid(h.double() @ sg.double().T).flatten()) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,F,E,I,top,shared,T", [(64, 24, 6, 2, 2, 32, 37), (100, 14, 5, 0, 1, 0, 9), (64, 8, 2, 6, 5, 16, 50),
                                                  (128, 64, 8, 3, 3, 48, 300), (64, 16, 1, 3, 1, 24, 40)])
def test_routed_feed_forward_alone(dtype, W, F, E, I, top, shared, T):
    """The whole part against the plain one: identity experts, the gated shared expert behind its gate, any number of rows."""
    from llm_b200.engine.context import Workspace
    from llm_b200.models.kepevik import _ffn
    from llm_b200.parts.base import build_part
    spec = _ffn(SimpleNamespace(width=W), {"kind": "moe", "ff": F, "experts": E, "identity": I, "top": top, "shared": shared}, "m")
    part = build_part("ffn", spec, DT[dtype], torch.device("cuda"))
    g = torch.Generator().manual_seed(W + E)
    infos = dict(part.parameters())
    for child in part.children():
        infos.update(child.parameters())
    w = {n: bf(torch.randn(info.shape, generator=g) * (0.2 if n.endswith("correction") else 1.3 / math.sqrt(info.shape[-1]))) for n, info in infos.items()}
    td = {n: dev(v, "float32" if infos[n].kind == "gain" else dtype) for n, v in w.items()}
    for q in [part] + list(part.children()):
        q.bind(td)
    x = bf(torch.randn(T, W, generator=g))
    mlp = {"router": {"experts": E, "identity": I, "top": top}, "shared": {"ff": shared} if shared else None}
    p = P.sub({k: v.double() for k, v in w.items()}, "m")
    ref, margin = P.moe_ff(x.double(), p, mlp), P.route(x.double(), p, mlp["router"])[2]
    ids = P.route(x.double(), p, mlp["router"])[0]
    assert I == 0 or bool((ids >= E).any()), "premise: some tokens choose an identity expert"
    ctx = SimpleNamespace(n_tokens=T, workspace=Workspace(max(T, 64), torch.device("cuda")), decode_only=False)
    out = part.forward(dev(x, dtype), ctx)
    late = part.forward(dev(x, dtype), ctx, allow_unsummed=True)
    resid = torch.zeros(T, W, device="cuda")
    from llm_b200.csrc import ops
    ops.add_rmsnorms(resid, late, None, 1.0, None, None, T, 1e-6)
    assert max_err(resid, out) < (1e-6 if dtype == "float32" else 8e-3)
    clear = margin > (1e-5 if dtype == "float32" else 1e-2)
    assert int(clear.sum()) > T // 2 and max_err(out[clear.cuda()], ref[clear]) < (2e-6 if dtype == "float32" else 1.5e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,dims,page", [(4, 2, 16, 8, 16), (3, 3, 10, 6, 8), (2, 1, 24, 0, 32), (8, 2, 64, 64, 16), (5, 1, 128, 32, 16)])
def test_values_stored_are_the_keys_before_rotation(dtype, H, G, D, dims, page):
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 100 + D)
    T, base = 40, 300.0
    qk = bf(torch.randn(T, (H + G) * D, generator=g))
    pos = [7 * t + 3 for t in range(T)]
    slots = torch.randperm(page * 6, generator=g)[:T].tolist()
    k_pages = torch.full((6, G, page, D), 9.0, device="cuda", dtype=DT[dtype])
    v_pages = torch.full((6, G, page, D), 9.0, device="cuda", dtype=DT[dtype])
    freqs = dev(torch.tensor([base ** (-2.0 * i / max(dims, 1)) for i in range(dims // 2)])) if dims else None
    q_out = torch.empty(T, H * D, device="cuda", dtype=DT[dtype])
    ops.norm_rope_kv_write(dev(qk, dtype), None, None, 1e-6, freqs, True, i32(pos), i32(slots), k_pages, v_pages, T, H, G, D, D,
                           q_out=q_out, v_from_k=True)
    turned = torch.zeros(max(pos) + 1, H + G, D, dtype=torch.float64)
    turned[pos] = qk.double().view(T, H + G, D)
    turned = P.rotate_halves(turned, dims, base)[pos]
    assert max_err(q_out, turned[:, :H].reshape(T, H * D)) < max(KTOL[dtype], 2e-5)
    for t, s in enumerate(slots):
        assert max_err(k_pages[s // page, :, s % page], turned[t, H:]) < max(KTOL[dtype], 1e-4)
        assert torch.equal(v_pages[s // page, :, s % page].cpu().float(), qk[t, H * D:].view(G, D))


MLSTM_SIZES = [(1, 4, 4), (2, 16, 24), (3, 10, 6), (3, 48, 56), (4, 32, 72), (1, 100, 130), (2, 128, 128), (1, 256, 8), (5, 7, 67)]


def _mlstm_inputs(T, H, D, V, seed, spread=2.0, mean_f=1.5):
    g = torch.Generator().manual_seed(seed)
    q, k, v = (bf(torch.randn(T, H * n, generator=g)) for n in (D, D, V))
    z = torch.randn(T, 2 * H, generator=g) * spread
    z[:, H:] += mean_f
    return q, k, v, z, torch.randn(H, generator=g), torch.randn(H, generator=g)


def _plain_mlstm(q, k, v, z, ib, fb, cap, H, D, V):
    T = q.shape[0]
    p = {"i": torch.eye(2 * H, dtype=torch.float64)[:H], "f": torch.eye(2 * H, dtype=torch.float64)[H:], "i.b": ib.double(), "f.b": fb.double()}
    i, f = P.mlstm_gates(z.double(), p, cap)
    return P.mlstm_scan(q.double().view(T, H, D) * D ** -0.5, k.double().view(T, H, D), v.double().view(T, H, V), i, f).reshape(T, H * V)


def _mlstm_steps(seq, cap, H, D, V, cuts, state, slot, forms, other_slot=None):
    """Run a request's tokens through its slot in portions; forms(n) names the kernel for a portion of n tokens: 'single', 'scan'
    or 'chunks'.  A single token of another request stands in front of every portion if other_slot is given."""
    from llm_b200.csrc import ops
    q, k, v, z, ib, fb = seq
    T = q.shape[0]
    out = torch.empty(T, H * V, device="cuda")
    gates = (dev(ib), dev(fb), cap, D ** -0.5, state)
    for a, b in split_steps(T, cuts):
        lead = 0 if other_slot is None else 1
        ctx = step_ctx([1] * lead + [b - a], ([other_slot] if lead else []) + [slot])
        cat = lambda t: torch.cat([t[:lead], t[a:b]])
        o = torch.empty(lead + b - a, H * V, device="cuda")
        form = forms(b - a)
        if form == "chunks":
            qkv = dev(torch.cat([cat(q), cat(k), cat(v)], dim=1), "bfloat16")
            n = ops.mlstm_chunk_scratch(ctx.n_tokens // 64 + ctx.n_entries, H, D, V)
            ops.mlstm_chunks(o, qkv[:, :H * D], qkv[:, H * D:2 * H * D], qkv[:, 2 * H * D:], dev(cat(z)), *gates, ctx, H, D, V,
                             [torch.full((m,), float("nan"), device="cuda") for m in n])
        else:
            proj = dev(torch.cat([cat(q), cat(k), cat(v), cat(v), cat(z)], dim=1))
            ops.mlstm_scan(o, proj, 2 * H * (D + V), *gates, ctx, H, D, V, single=form == "single" and b - a == 1)
        out[a:b] = o[lead:]
    return out


@pytest.mark.parametrize("H,D,V", MLSTM_SIZES)
@pytest.mark.parametrize("cap", [1.5, 12.5])
def test_matrix_memory_in_steps_equals_the_plain_loop(H, D, V, cap):
    """Portions token by token, single tokens by their own kernel where it takes the sizes, beside another request's token."""
    from llm_b200.csrc import ops
    T = 150
    seq = _mlstm_inputs(T, H, D, V, H * 1000 + D)
    ref = _plain_mlstm(*seq, cap, H, D, V)
    state = torch.zeros(4, ops.mlstm_state(H, D, V)[2], device="cuda")
    single = ops.mlstm_single_available(D, V, state)
    out = _mlstm_steps(seq, cap, H, D, V, (40, 1, 2, 17, 1, 1, 33), state, 2, lambda n: "single" if single else "scan", other_slot=0)
    assert max_err(out, ref) < 3e-5
    assert float(state[1].abs().max()) == 0 and float(state[3].abs().max()) == 0
    state.zero_()
    out = _mlstm_steps(seq, cap, H, D, V, (1,), state, 3, lambda n: "single" if single else "scan")
    assert max_err(out, ref) < 3e-5


@pytest.mark.parametrize("H,D,V", [s for s in MLSTM_SIZES if s[1] % 16 == 0 and s[2] % 8 == 0] + [(3, 64, 40), (2, 32, 200), (1, 80, 64)])
@pytest.mark.parametrize("cap", [1.5, 12.5])
def test_matrix_memory_chunk_by_chunk_equals_the_plain_loop(H, D, V, cap):
    """Portions off every chunk border, from states that other forms left, and the state handed back to those forms.  (A chunk's
    log gates are sums of up to 64 numbers of the cap's size, so their exponentials carry a few 1e-5 of rounding.)"""
    from llm_b200.csrc import ops
    T = 460
    seq = _mlstm_inputs(T, H, D, V, H * 1000 + D + 3)
    ref = _plain_mlstm(*seq, cap, H, D, V)
    state = torch.zeros(4, ops.mlstm_state(H, D, V)[2], device="cuda")
    out = _mlstm_steps(seq, cap, H, D, V, (63, 1, 129, 2, 64, 1, 190), state, 1, lambda n: "chunks" if n > 2 else "single" if n == 1 else "scan")
    assert max_err(out, ref) < 1e-4
    walked = torch.zeros_like(state)
    _mlstm_steps(seq, cap, H, D, V, (T,), walked, 1, lambda n: "scan")
    assert max_err(state, walked) < 1e-4 and float(state[0].abs().max()) == 0
    # every copy of n and m is alike
    n_off, m_off, size = ops.mlstm_state(H, D, V)
    blocks = -(-V // 64)
    n = state[1, n_off:n_off + H * blocks * D].view(H, blocks, D)
    m = state[1, m_off:m_off + H * blocks].view(H, blocks)
    assert torch.equal(n, n[:, :1].expand_as(n)) and torch.equal(m, m[:, :1].expand_as(m))


def test_running_maximum_starts_at_zero_and_the_floor_holds():
    """Input gates far below zero: the memory is then small beside exp(-m), which must come from the maximum's start at zero; with
    forget gates near one the denominator stays the floor for the whole request."""
    H, D, V, T, cap = 2, 16, 24, 200, 30.0
    q, k, v, z, ib, fb = _mlstm_inputs(T, H, D, V, 5, spread=0.5, mean_f=12.0)
    ib = torch.full((H,), -8.0)
    ref = _plain_mlstm(q, k, v, z, ib, fb, cap, H, D, V)
    i, f = P.mlstm_gates(z.double(), {"i": torch.eye(2 * H).double()[:H], "f": torch.eye(2 * H).double()[H:], "i.b": ib.double(), "f.b": fb.double()}, cap)
    late = P.mlstm_scan(q.double().view(T, H, D) * D ** -0.5, k.double().view(T, H, D), v.double().view(T, H, V),
                        i + 40.0, f).reshape(T, H * V)          # gates so large that the start no longer matters
    assert float((late - ref).abs().max() / late.abs().max()) > 0.3, "premise: the floor matters"
    from llm_b200.csrc import ops
    for forms in (lambda n: "scan", lambda n: "chunks"):
        state = torch.zeros(2, ops.mlstm_state(H, D, V)[2], device="cuda")
        out = _mlstm_steps((q, k, v, z, ib, fb), cap, H, D, V, (150, 50), state, 1, forms)
        assert max_err(out, ref) < 3e-5


DELTA_SIZES = [(1, 1, 4, 4), (4, 2, 16, 8), (3, 3, 12, 10), (4, 1, 64, 32), (2, 2, 100, 36), (2, 1, 128, 64), (1, 1, 256, 5), (6, 2, 8, 130)]


def _delta_inputs(T, H, G, D, V, seed, fast=False):
    g = torch.Generator().manual_seed(seed)
    q, k = bf(torch.randn(T, G * D, generator=g)), bf(torch.randn(T, G * D, generator=g))
    v, b = bf(torch.randn(T, H * V, generator=g)), bf(torch.randn(T, H, generator=g))
    z = torch.randn(T, H * D, generator=g) * (3.0 if fast else 1.0)
    a_log, dt_bias = torch.randn(H, generator=g) * 0.7 + (1.5 if fast else -1.0), torch.randn(H * D, generator=g) * 1.5 - 1.0
    return q, k, v, b, z, a_log, dt_bias


def _plain_delta(q, k, v, b, z, a_log, dt_bias, H, G, D, V):
    T = q.shape[0]
    of = torch.tensor([P.kv_head_of(h, H, G) for h in range(H)])
    q, k = P.unit(q.double().view(T, G, D)) * D ** -0.5, P.unit(k.double().view(T, G, D))
    decay = torch.exp(-torch.exp(a_log.double()).view(1, H, 1) * P.softplus(z.double() + dt_bias.double()).view(T, H, D))
    return P.delta_scan(q[:, of], k[:, of], v.double().view(T, H, V), torch.sigmoid(b.double()), decay).reshape(T, H * V)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,V", DELTA_SIZES)
def test_channel_decayed_delta_rule_in_steps_equals_the_plain_loop(dtype, H, G, D, V):
    from llm_b200.csrc import ops
    T = 150
    q, k, v, b, z, a_log, dt_bias = _delta_inputs(T, H, G, D, V, H * 1000 + D)
    ref = _plain_delta(q, k, v, b, z, a_log, dt_bias, H, G, D, V)
    state = torch.zeros(4, H * D * V, device="cuda")
    out = torch.empty(T, H * V, device="cuda")
    for s, e in split_steps(T, (40, 1, 2, 17, 1, 33)):
        ctx = step_ctx([1, e - s], [3, 1])
        cat = lambda t: torch.cat([t[:1], t[s:e]])
        qk = dev(torch.cat([cat(q), cat(k)], dim=1), dtype)
        o = torch.empty(1 + e - s, H * V, device="cuda")
        ops.delta_scan(o, qk[:, :G * D], qk[:, G * D:], dev(cat(v), dtype), dev(cat(b), dtype), dev(cat(z)), dev(a_log), dev(dt_bias), state,
                       ctx, H, G, D, V, D ** -0.5, per_channel=True)
        out[s:e] = o[1:]
    assert max_err(out, ref) < 3e-5
    assert float(state[0].abs().max()) == 0 and float(state[2].abs().max()) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,V", DELTA_SIZES)
@pytest.mark.parametrize("fast", [False, True])
def test_channel_decayed_delta_rule_chunk_by_chunk_equals_the_plain_loop(dtype, H, G, D, V, fast):
    """A step of four entries (one token, portions off every chunk and block border, a long one) from non-zero states; fast: decays
    that fall to nothing within a few tokens on some channels, where a plain quotient of decays would overflow."""
    from llm_b200.csrc import ops
    lens, T0 = [1, 77, 13, 300], 40
    state = torch.zeros(5, H * D * V, device="cuda")
    seqs, refs = [], []
    for e, n in enumerate(lens):       # every entry: T0 earlier tokens token by token (the state it starts from), then the step
        seq = _delta_inputs(T0 + n, H, G, D, V, H * 1000 + D + 7 + e, fast)
        if e:
            seq = seq[:5] + (a_log, dt_bias)
        q, k, v, b, z, a_log, dt_bias = seq
        refs.append(_plain_delta(*seq, H, G, D, V)[T0:])
        seqs.append(seq)
        ops.delta_scan(torch.empty(T0, H * V, device="cuda"), dev(q[:T0], dtype), dev(k[:T0], dtype), dev(v[:T0], dtype), dev(b[:T0], dtype),
                       dev(z[:T0]), dev(a_log), dev(dt_bias), state, step_ctx([T0], [e + 1]), H, G, D, V, D ** -0.5, per_channel=True)
    cat = lambda i: dev(torch.cat([sq[i][T0:] for sq in seqs]), "float32" if i == 4 else dtype)
    T = sum(lens)
    ctx = step_ctx(lens, [1, 2, 3, 4])
    out = torch.empty(T, H * V, device="cuda")
    scratch = [torch.full((n,), float("nan"), device="cuda") for n in ops.delta_chunk_scratch(T // 32 + len(lens), H, D, V, True)]
    walked = state.clone()
    rest = (dev(a_log), dev(dt_bias))
    ops.delta_chunk_scan(out, cat(0), cat(1), cat(2), cat(3), cat(4), *rest, state, ctx, H, G, D, V, D ** -0.5, 1e-6, scratch, per_channel=True)
    assert max_err(out, torch.cat(refs)) < 3e-5
    out2 = torch.empty(T, H * V, device="cuda")
    ops.delta_scan(out2, cat(0), cat(1), cat(2), cat(3), cat(4), *rest, walked, ctx, H, G, D, V, D ** -0.5, per_channel=True)
    assert max_err(state, walked) < 3e-5 and float(state[0].abs().max()) == 0


# ---- whole models ---------------------------------------------------------------------
LENGTHS = {"A": [1, 5, 33, 70, 129], "B": [2, 47, 64, 150, 260], "C": [3, 40, 17, 90], "D": [1, 16, 130, 200], "E": [1, 130, 31, 257],
           "F": [2, 33, 140, 95], "G": [1, 2, 60, 75]}
MARGIN = 0.02      # bfloat16: a choice of experts that hangs on less than this may fall otherwise


def plain(cfg, w, toks, margins=None):
    return P.forward(cfg, {k: v.double() for k, v in w.items()}, toks, margins=margins)


def clear_rows(cfg, w, toks):
    """Rows before the first token whose routing is a close call: after it a bfloat16 engine may have chosen other experts,
    and every later token inherits the difference through attention or state."""
    margins = []
    plain(cfg, w, toks, margins=margins)
    if not margins:
        return len(toks)
    close = torch.nonzero(torch.stack(margins).min(dim=0).values < MARGIN).flatten()
    return int(close[0]) if close.numel() else len(toks)


@pytest.fixture(scope="module")
def models():
    cache = {}

    def get(name):
        if name not in cache:
            cfg, page = CONFIGS[name]
            w = make_weights(cfg, seed=ord(name), slow=3.0 if name == "F" else 0.0)
            reqs = {f"r{i}": random_tokens(n, cfg["vocab"], 300 + i) for i, n in enumerate(LENGTHS[name])}
            ref = {rid: plain(cfg, w, toks) for rid, toks in reqs.items()}
            upto = {rid: clear_rows(cfg, w, toks) for rid, toks in reqs.items()}
            cache[name] = (cfg, page, w, reqs, ref, upto)
        return cache[name]
    return get


def compare(got, ref, dtype, what, upto=None, tol=None, strict=None):
    """Every row's largest difference, relative to the request's largest logit, against the bound of the dtype.  float32:
    every row.  bfloat16: the rows before a request's first close routing call (upto), of which one in fifty (at least one) may
    pass the bound, up to half the largest logit; the rows named in `strict` may not."""
    tol = tol or TOL[dtype]
    for rid, r in ref.items():
        assert got[rid].shape == r.shape, f"{what}: {rid} shape {got[rid].shape} vs {r.shape}"
        err_rows = (got[rid].double() - r).abs().max(dim=1).values / r.abs().max()
        assert bool(torch.isfinite(err_rows).all()), f"{what}: request {rid} has rows that are not finite"
        if dtype == "bfloat16" and upto is not None:
            err_rows = err_rows[:upto[rid]]
            if not err_rows.numel():
                continue
        bad = torch.nonzero(~(err_rows <= tol)).flatten()
        first = f"{what}: request {rid} first differs at position {int(bad[0]) if bad.numel() else -1} " \
                f"(err {float(err_rows.max()):.3e} at most, limit {tol:.1e})"
        if strict:
            assert float(err_rows[strict].max()) <= tol, first
        if dtype == "float32":
            assert bad.numel() == 0, first
        else:
            assert bad.numel() <= max(1, len(err_rows) // 50) and float(err_rows.max()) <= 0.5, first


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_cut_matches_plain(models, name, dtype):
    cfg, page, w, reqs, ref, upto = models(name)
    longest = max(len(t) for t in reqs.values())
    eng = make_engine(cfg, w, dtype, page, -(-longest // page) + 1)       # a pool barely larger than the longest request
    compare(replay.run_steps(eng, replay.steps_whole(reqs)), ref, dtype, "whole", upto)
    compare(replay.run_steps(eng, replay.steps_tail_decode(reqs)), ref, dtype, "tail decode", upto)
    compare(replay.run_steps(eng, replay.steps_portions(reqs)), ref, dtype, "portions", upto)
    compare(replay.run_steps(eng, replay.steps_portions(reqs, sizes=(2, 2, 3, 2, 16, 2, 17, 64))), ref, dtype, "small portions", upto)
    eng.check_status()
    eng.cache.check()
    assert all(eng.cache.num_free_pages(g) == eng.cache.group_spec(g).num_pages for g in range(eng.cache.num_groups))
    lens = sorted((len(t) for t in reqs.values()), reverse=True)
    eng = make_engine(cfg, w, dtype, page, sum(-(-n // page) for n in lens[:4]) + 1)
    compare(replay.run_steps(eng, replay.steps_mixed(reqs)), ref, dtype, "mixed", upto)     # freed pages and slots are used again
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_batch_of_unequal_requests_equals_each_alone(models, name, dtype):
    from llm_b200.engine.engine import StepEntry
    cfg, page, w, reqs, ref, upto = models(name)
    eng = make_engine(cfg, w, dtype, page, 60)
    alone = replay.run_steps(eng, replay.steps_whole(reqs))
    entries = [StepEntry(rid, toks, list(range(len(toks)))) for rid, toks in reqs.items()][:4]
    rows = eng.step(entries).float().cpu()
    at = 0
    for e in entries:
        n = len(e.tokens)
        m = n if dtype == "float32" else upto[e.request_id]
        if m:
            assert max_err(rows[at:at + m], alone[e.request_id][:m]) < (1e-5 if dtype == "float32" else 2e-2)
        at += n
        eng.release(e.request_id)


def test_pages_and_slots_go_back_and_are_used_again():
    """Many requests one after another through a pool that holds one of them and one state slot."""
    cfg, page = CONFIGS["E"]
    w = make_weights(cfg, seed=5)
    reqs = {f"r{i}": random_tokens(n, cfg["vocab"], 40 + i) for i, n in enumerate([96, 33, 64, 96, 5])}
    ref = {rid: plain(cfg, w, toks) for rid, toks in reqs.items()}
    eng = make_engine(cfg, w, "float32", page, 3, max_tokens=48, max_seqs=1, max_seq_len=96)
    compare(replay.run_steps(eng, replay.steps_portions(reqs, sizes=(40, 2, 31, 1, 16, 48))), ref, "float32", "portions")
    eng.cache.check()
    assert eng.cache.num_free_pages(0) == 3


# ---- keys far away and at page borders ----------------------------------------------------------------
NEEDLE, QUERY = 7, 11


def _far_key_model(kv_heads, dim=32):
    """The attention alone (the delta rule beside it is scaled by zero, there is no feed-forward, nothing turns) whose head 0
    sends the token QUERY to the token NEEDLE: the needle's embedding is solved for, so that its key points where the query of
    QUERY points and the pair scores several deviations above every other one.  The embedding is small beside what the mixer
    writes."""
    cfg = config(64, 80, 2.0, [layer(parallel(2, kv_heads, dim, 0.25, 0, 100.0, r_heads=1, r_kv=1, r_dim=8, r_vdim=8, r_conv=2,
                                              left_scale=1.0, right_scale=0.0), None)])
    w = make_weights(cfg, seed=11 + kv_heads, peak=4.0)
    w["embed"] = w["embed"] * 0.25
    w["l0.norm1"] = torch.zeros(64)
    q = w["l0.mix.left.q"][:dim].double() @ P.rms_unit(w["embed"][QUERY].double(), 0.0)
    needle = torch.linalg.pinv(w["l0.mix.left.k"][:dim].double()) @ q
    w["embed"][NEEDLE] = (needle * w["embed"][QUERY].norm() / needle.norm()).to(torch.bfloat16).float()
    return cfg, w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kv_heads,p", [(1, 5), (2, 15), (1, 16), (2, 31), (1, 0)])
def test_attention_finds_a_key_hundreds_of_tokens_back(dtype, kv_heads, p):
    """One NEEDLE near the start (the first token and the ends of pages among the places), QUERY tokens hundreds of tokens later;
    the rows of the queries change when the needle is exchanged (plain side), and those are the strict ones."""
    cfg, w = _far_key_model(kv_heads)
    T, asks = 700, [400, 511, 512, 699]
    toks = [t if t not in (NEEDLE, QUERY) else t + 20 for t in random_tokens(T, cfg["vocab"], 3)]
    toks[p] = NEEDLE
    for i in asks:
        toks[i] = QUERY
    other = list(toks)
    other[p] = 33
    ref, ref_other = plain(cfg, w, toks), plain(cfg, w, other)
    moved = (ref - ref_other).abs().max(dim=1).values / ref.abs().max()
    assert float(moved[asks].min()) > 0.06, "premise: the far rows hang on the exchanged token"
    tol = None if dtype == "float32" else 3e-2
    eng = make_engine(cfg, w, dtype, 16, -(-T // 16) + 1, max_tokens=704)
    compare(replay.run_steps(eng, replay.steps_whole({"x": toks})), {"x": ref}, dtype, "whole", strict=asks, tol=tol)
    compare(replay.run_steps(eng, replay.steps_tail_decode({"x": toks}, tail=380)), {"x": ref}, dtype, "decode", strict=asks, tol=tol)
    compare(replay.run_steps(eng, replay.steps_portions({"x": toks}, sizes=(100, 2, 37, 128, 3)), ), {"x": ref}, dtype, "portions", strict=asks, tol=tol)
    compare(replay.run_steps(eng, replay.steps_whole({"y": other})), {"y": ref_other}, dtype, "exchanged", strict=asks, tol=tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["mlstm", "delta"])
def test_state_remembers_a_token_from_hundreds_back(dtype, kind):
    """Slow decays; the request's state slot was another request's before; portions cut the sequence everywhere."""
    if kind == "mlstm":
        cfg = config(48, 70, 1.0, [layer(mlstm(2, 16, 24, 9.0), None)])
    else:
        cfg = config(48, 70, 1.0, [layer(parallel(1, 1, 8, 0.3, 4, 100.0, r_heads=2, r_kv=1, r_dim=16, r_vdim=24, r_conv=3,
                                                  left_scale=0.0, right_scale=1.0), None)])
    w = make_weights(cfg, seed=9, slow=6.0)
    if kind == "delta":
        w["l0.mix.right.b"] = w["l0.mix.right.b"] * 0.0                # beta = 1/2 everywhere: every token writes
        w["l0.mix.right.dt_bias"] = torch.full((32,), -6.0)
        w["l0.mix.right.A_log"] = torch.full((2,), -3.0)
    else:
        w["l0.mix.f.b"] = torch.full((2,), 8.0)
    T, p = 700, 20
    toks = random_tokens(T, cfg["vocab"], 5)
    other = list(toks)
    other[p] = (toks[p] + 9) % cfg["vocab"]
    ref, ref_other = plain(cfg, w, toks), plain(cfg, w, other)
    moved = (ref - ref_other).abs().max(dim=1).values / ref.abs().max()
    assert float(moved[650:].max()) > 1e-3, "premise: the state still holds the exchanged token"      # float32 sees 3e-5
    eng = make_engine(cfg, w, dtype, 16, 50, max_tokens=256, max_seqs=2)
    first = replay.run_steps(eng, replay.steps_whole({"warm": random_tokens(90, cfg["vocab"], 1)}))      # uses and frees a slot
    got = replay.run_steps(eng, replay.steps_portions({"x": toks}, sizes=(100, 2, 64, 1, 200, 31)))
    tol = None if dtype == "float32" else 8e-2
    compare(got, {"x": ref}, dtype, "portions", tol=tol)
    got = replay.run_steps(eng, replay.steps_portions({"y": other}, sizes=(128,)))
    compare(got, {"y": ref_other}, dtype, "exchanged", tol=tol)
    assert first["warm"].shape[0] == 90


def test_a_slot_that_is_used_again_starts_from_zero(models):
    cfg, page, w, reqs, ref, upto = models("A")
    eng = make_engine(cfg, w, "float32", page, 40, max_seqs=1)           # one slot: every request takes the same one
    for _ in range(2):
        compare(replay.run_steps(eng, replay.steps_whole(reqs)), ref, "float32", "whole, one slot")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_long_decode_with_graphs_and_first_tokens(models, name, dtype):
    """One prompt token, then 210 decoded one by one under CUDA graphs, beside a second request that joins late."""
    cfg, page = CONFIGS[name]
    w = make_weights(cfg, seed=77)
    toks, late = random_tokens(211, cfg["vocab"], 21), random_tokens(40, cfg["vocab"], 22)
    ref = {"x": plain(cfg, w, toks), "late": plain(cfg, w, late)}
    upto = {"x": clear_rows(cfg, w, toks), "late": clear_rows(cfg, w, late)}
    eng = make_engine(cfg, w, dtype, page, 40, graphs=True)
    steps = []
    for i in range(len(toks)):
        entries = [{"id": "x", "tokens": toks[i:i + 1], "want": [0]}]
        j = i - 100
        if 0 <= j < len(late):
            entries.append({"id": "late", "tokens": late[j:j + 1], "want": [0]})
        steps.append({"entries": entries, "end": []})
    steps[-1]["end"] = ["x", "late"]
    compare(replay.run_steps(eng, steps), ref, dtype, "decode from the first token", upto)
    eng.check_status()


def test_prefill_equals_token_by_token_from_the_first_token(models):
    for name in ("A", "E", "G"):
        cfg, page = CONFIGS[name]
        w = make_weights(cfg, seed=31)
        toks = random_tokens(70, cfg["vocab"], 6)
        eng = make_engine(cfg, w, "float32", page, 20)
        whole = replay.run_steps(eng, replay.steps_whole({"x": toks}))["x"]
        single = replay.run_steps(eng, replay.steps_tail_decode({"x": toks}, tail=69))["x"]
        assert max_err(single, whole) < 2e-5


def _plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(plain(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """LLM.generate: the scheduler admits, batches, pages and samples; greedy tokens equal the plain implementation's."""
    from llm_b200 import LLM
    cfg, page = CONFIGS["A"]
    w = make_weights(cfg, seed=41)
    prompts = [random_tokens(n, cfg["vocab"], 500 + n) for n in (1, 9, 30, 47, 18)]
    llm = LLM(None, dtype="float32", max_num_seqs=3, max_num_batched_tokens=16, kv_block_size=page, num_kv_blocks=14,
              eos_token_id=-1, random_config=cfg, tensors={k: v.clone() for k, v in w.items()}, max_seq_len=128)
    got = llm.generate(prompts, max_new_tokens=16)
    for p, g in zip(prompts, got):
        assert g == _plain_greedy(cfg, w, p, 16)
    llm.engine.cache.check()


def test_trace_replay_of_a_folder(models, tmp_path):
    """The trace runner on a folder written to disk in bfloat16: steps in, logit files out."""
    import io
    import numpy as np
    from llm_b200.engine import trace
    from llm_b200.weights.safetensors_io import write_safetensors
    cfg, page = CONFIGS["B"]
    w = make_weights(cfg, seed=51)
    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(d / "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in w.items()})
    reqs = {"a": random_tokens(70, cfg["vocab"], 1), "b": random_tokens(45, cfg["vocab"], 2)}
    steps = replay.steps_mixed(reqs, max_live=2)
    lines = "\n".join(json.dumps({"step": i, "entries": s["entries"], "end": s["end"]}) for i, s in enumerate(steps))
    out, said = tmp_path / "out", io.StringIO()
    assert trace.main(["--model", str(d), "--dtype", "float32", "--out", str(out), "--max-tokens", "128"], stdin=io.StringIO(lines),
                      stdout=said) == 0
    assert said.getvalue().split() == [x for i in range(len(steps)) for x in ("done", str(i))]
    rows = {}
    for i, s in enumerate(steps):
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
        at = 0
        for e in s["entries"]:
            rows.setdefault(e["id"], []).append(got[at:at + len(e["want"])])
            at += len(e["want"])
    got = {rid: torch.cat(parts) for rid, parts in rows.items()}
    compare(got, {rid: plain(cfg, w, toks) for rid, toks in reqs.items()}, "float32", "trace replay")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(10))
def test_seeded_random_configurations(seed, dtype):
    cfg = random_config(seed)
    page = [8, 16, 32][seed % 3]
    w = make_weights(cfg, seed=1000 + seed)
    reqs = {f"r{i}": random_tokens(n, cfg["vocab"], seed * 10 + i) for i, n in enumerate([1, 37, 120, 64])}
    ref = {rid: plain(cfg, w, toks) for rid, toks in reqs.items()}
    upto = {rid: clear_rows(cfg, w, toks) for rid, toks in reqs.items()}
    tol = 1e-4 if dtype == "float32" else 8e-2          # corner sizes and harsh constants among the drawn ones
    eng = make_engine(cfg, w, dtype, page, -(-120 // page) + 1)
    compare(replay.run_steps(eng, replay.steps_whole(reqs)), ref, dtype, f"seed {seed} whole", upto, tol=tol)
    compare(replay.run_steps(eng, replay.steps_tail_decode(reqs, tail=20)), ref, dtype, f"seed {seed} tail decode", upto, tol=tol)
    eng = make_engine(cfg, w, dtype, page, sum(-(-n // page) for n in (37, 120, 64)) + 2)
    compare(replay.run_steps(eng, replay.steps_mixed(reqs)), ref, dtype, f"seed {seed} mixed", upto, tol=tol)
    eng.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(4))
def test_seeded_configurations_of_layer_like_sizes(seed, dtype):
    cfg = random_config(100 + seed, large=True)
    w = make_weights(cfg, seed=2000 + seed)
    reqs = {f"r{i}": random_tokens(n, cfg["vocab"], seed * 10 + i) for i, n in enumerate([150, 40, 300])}
    ref = {rid: plain(cfg, w, toks) for rid, toks in reqs.items()}
    upto = {rid: clear_rows(cfg, w, toks) for rid, toks in reqs.items()}
    tol = 1e-4 if dtype == "float32" else 8e-2
    eng = make_engine(cfg, w, dtype, 16, 40)
    compare(replay.run_steps(eng, replay.steps_whole(reqs)), ref, dtype, f"seed {seed} whole", upto, tol=tol)
    compare(replay.run_steps(eng, replay.steps_mixed(reqs, prefill_sizes=(64, 2, 130, 17))), ref, dtype, f"seed {seed} mixed", upto, tol=tol)
    eng.check_status()
