"""GPU tests of the Nidorax design against the plain implementation (tests/plain_nidorax.py): each mechanism alone,
then whole models under every way of cutting the work."""
import json
import math
from types import SimpleNamespace

import pytest
import torch

import plain_nidorax as P
import replay
from nidorax_tiny import CONFIGS, config, latent, layer, lightning, make_engine, make_weights, moe, random_config, yarn
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


def partials_of(x, splits, g):
    """x as the unsummed partial results of a split-K product, in a PartialSum."""
    from llm_b200.csrc import ops
    parts = torch.randn(splits, *x.shape, generator=g)
    parts[-1] = x - parts[:-1].sum(dim=0)
    return parts.cuda().contiguous(), lambda buf, dtype: ops.PartialSum(buf, splits, x.shape[0], x.shape[1], dtype)


# ---- each mechanism alone ---------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,rows", [(64, 5), (100, 3), (2048, 4), (4096, 2), (8192, 2), (9000, 2), (17, 9)])
def test_norm_behind_the_sum(dtype, width, rows):
    """x <- rms(alpha x + y) (1 + w) from a tensor, from split-K partials and from the weighted rows of a routed feed-forward."""
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    x, w, alpha, eps = torch.randn(rows, width, generator=g), bf(torch.randn(width, generator=g) * 0.2), 1.7, 1e-3
    y = bf(torch.randn(rows, width, generator=g))
    gain = dev(w + 1.0)

    def run(term):
        resid = dev(x)
        out = None if dtype == "float32" else torch.empty(rows, width, device="cuda", dtype=DT[dtype])
        ops.sum_rmsnorm(resid, alpha, term, gain, out, rows, eps, DT[dtype])
        return resid, out

    def check(resid, out, y):
        ref = P.centred_norm(alpha * x.double() + y.double(), w.double(), eps)
        assert max_err(resid, ref) < 2e-6
        if out is not None:
            assert max_err(out, ref) < KTOL["bfloat16"] and torch.equal(out, resid.to(torch.bfloat16))
    check(*run(dev(y, dtype)), y)
    buf, make = partials_of(y, 5, g)
    check(*run(make(buf, DT[dtype])), y)
    top, slots = 3, 40
    ys = torch.randn(slots, width, generator=g)
    place = torch.randint(0, slots, (rows, top), generator=g)
    place[0, 1] = -1                                         # a pair without a slot counts nothing
    wts = torch.rand(rows, top, generator=g)
    want = (ys[place.clamp(min=0)] * (wts * (place >= 0)).unsqueeze(-1)).sum(dim=1)
    check(*run(ops.WeightedRows(dev(ys), place.to(torch.int32).cuda(), dev(wts), top, rows)), want)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,rows", [(64, 5), (18, 3), (2048, 2), (4096, 2), (6144, 3), (8200, 2)])
def test_norm_over_all_heads_with_a_sigmoid_gate(dtype, n, rows):
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(n)
    x, w = torch.randn(rows, n, generator=g), torch.randn(n, generator=g)
    proj = bf(torch.randn(rows, n + 16, generator=g))
    ref = P.rms_norm(x.double(), w.double(), 1e-4) * torch.sigmoid(proj[:, 16:].double())
    out = torch.empty(rows, n, device="cuda", dtype=DT[dtype])
    ops.row_rmsnorm_sigmoid(out, dev(x), dev(w), dev(proj, dtype), 16, rows, 1e-4)
    assert max_err(out, ref) < KTOL[dtype]
    buf, make = partials_of(proj, 3, g)
    out.zero_()
    ops.row_rmsnorm_sigmoid(out, dev(x), dev(w), make(buf, DT[dtype]), 16, rows, 1e-4)
    assert max_err(out, ref) < KTOL[dtype]


@pytest.mark.parametrize("E,top,count,keep", [(8, 2, 2, 1), (6, 2, 3, 2), (5, 1, 5, 2), (3, 3, 1, 1), (20, 4, 5, 3), (37, 5, 1, 1), (16, 16, 4, 4),
                                              (256, 8, 8, 4), (64, 6, 64, 9)])
def test_softmax_router_chooses_among_the_best_groups(E, top, count, keep):
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(E * 10 + top)
    T, W = 50, 24
    h = bf(torch.randn(T, W, generator=g))
    p = {"router": bf(torch.randn(E, W, generator=g) * 0.5), "correction": bf(torch.randn(E, generator=g) * 0.1 - 0.2)}
    r = {"experts": E, "top": top, "groups": {"count": count, "keep": keep}}
    ids_ref, w_ref, margin = P.route(h.double(), {k: v.double() for k, v in p.items()}, r)
    logits = torch.empty(T, E, device="cuda")
    ids = torch.empty(T * top, dtype=torch.int32, device="cuda")
    wts = torch.empty(T * top, device="cuda")
    ops.moe_route(dev(h), dev(p["router"]), dev(p["correction"]), logits, ids, wts, T, top, groups=(count, keep), softmax=True, group_max=True,
                  renorm_eps=1e-20)
    ids, wts = ids.view(T, top).cpu().long(), wts.view(T, top).cpu()
    clear = margin > 1e-5
    assert int(clear.sum()) > T // 2
    assert torch.equal(ids[clear], ids_ref[clear])
    assert max_err(wts[clear], w_ref[clear]) < 1e-5 and max_err(wts.sum(dim=1), torch.ones(T)) < 1e-5


@pytest.mark.parametrize("W,heads,page", [(192, 2, 16), (256, 6, 8), (320, 16, 32), (384, 1, 16), (512, 20, 16), (576, 16, 16), (640, 33, 64)])
def test_attention_over_wide_latents(W, heads, page):
    """Ragged portions behind cached tokens, beside single tokens; then single tokens alone with the keys in one range and in
    several (an empty one among them); shuffled pages, unused rows poisoned.  One key a row stands far out."""
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(W + heads)
    held, new = [150, 65, 1, 300, 33], [150, 1, 1, 90, 32]
    E, scale = len(held), 0.7 / math.sqrt(W)
    c = bf(torch.randn(E, max(held), W, generator=g))
    q = bf(torch.randn(sum(new), heads, W, generator=g))
    for r in range(0, sum(new), 5):                                   # these rows ask for one key, at different distances
        e = max(i for i in range(E) if sum(new[:i]) <= r)
        pos = held[e] - new[e] + r - sum(new[:e])
        q[r] = bf(3.0 * c[e, (r * 37) % (pos + 1)])
    per = -(-max(held) // page)
    perm = torch.randperm(E * per + 2, generator=g)[:E * per].view(E, per)
    pages = torch.full((E * per + 2, 1, page, W), float("nan"))
    for e in range(E):
        for t in range(held[e]):
            pages[perm[e, t // page], 0, t % page] = c[e, t]
    ref, cu = [], [0]
    for e in range(E):
        for i in range(new[e]):
            n = held[e] - new[e] + i + 1
            s = torch.softmax(q[cu[e] + i].double() @ c[e, :n].double().T * scale, dim=1)
            ref.append((s @ c[e, :n].double()).flatten())
        cu.append(cu[-1] + new[e])
    ref = torch.stack(ref)
    pd, table, qd = dev(pages, "bfloat16"), perm.to(torch.int32).cuda().contiguous(), dev(q.view(-1, heads * W), "bfloat16")
    out = torch.full_like(qd, float("nan"))
    ops.attention_wide(out, qd, pd, table, i32(cu), i32(held), cu[-1], E, heads, scale)
    assert max_err(out, ref) < 1.2e-2          # P is rounded to bfloat16 before the second product
    last = [n - 1 for n in cu[1:]]
    for splits in (1, 2, 7, 0):
        out = torch.full((E, heads * W), float("nan"), device="cuda", dtype=torch.bfloat16)
        ops.attention_wide(out, qd[last].contiguous(), pd, table, i32(list(range(E + 1))), i32(held), E, E, heads, scale, decode=True,
                           max_keys=max(held), splits=splits)
        assert max_err(out, ref[last]) < 1.2e-2


@pytest.mark.parametrize("D,heads,parts", [(128, 16, 1), (128, 16, 4), (64, 24, 2), (128, 32, 2), (64, 40, 8), (128, 6, 3)])
@pytest.mark.parametrize("splits", [1, 3, 12])
def test_decode_attention_with_the_heads_of_a_latent_split_over_ctas(D, heads, parts, splits):
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(D + heads)
    page, lens, scale = 16, [333, 70, 16, 1], 0.15
    c = bf(torch.randn(len(lens), max(lens), D, generator=g))
    q = bf(torch.randn(len(lens), heads * D, generator=g))
    per = -(-max(lens) // page)
    perm = torch.randperm(len(lens) * per, generator=g).view(len(lens), per)
    pages = torch.zeros(len(lens) * per, 1, page, D)
    for e in range(len(lens)):
        for t in range(lens[e]):
            pages[perm[e, t // page], 0, t % page] = c[e, t]
    ref = torch.zeros(len(lens), heads, D, dtype=torch.float64)
    for e, n in enumerate(lens):
        s = torch.softmax(q[e].view(heads, D).double() @ c[e, :n].double().T * scale, dim=1)
        ref[e] = s @ c[e, :n].double()
    out = torch.empty(len(lens), heads * D, device="cuda", dtype=torch.bfloat16)
    pd = dev(pages, "bfloat16")
    for _ in range(2):                      # the arrival counters are zero again after a launch
        ops.paged_attention_decode(out, dev(q, "bfloat16"), pd, pd, perm.to(torch.int32).cuda().contiguous(), i32(lens), len(lens), heads, 1, D, 0,
                                   scale, splits=splits, max_keys=max(lens), head_parts=parts)
        assert max_err(out, ref.view(len(lens), -1)) < 1e-2


@pytest.mark.parametrize("tile", [16, 32, 128])
@pytest.mark.parametrize("T,top,E,W,F", [(1, 2, 4, 64, 72), (8, 4, 16, 256, 200), (40, 3, 5, 128, 96), (64, 2, 3, 72, 136), (5, 1, 1, 2048, 1408)])
def test_expert_products_in_tiles_of_few_rows(tile, T, top, E, W, F):
    """Rows sorted by expert into tiles of 16, 32 or 128 slots, an expert's run over several tiles among them: up-projection with
    the squared relu in the epilogue, then the down-projection into float32."""
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(T * 100 + tile)
    x, up, down = bf(torch.randn(T, W, generator=g)), bf(torch.randn(E, F, W, generator=g) / math.sqrt(W)), bf(torch.randn(E, W, F, generator=g) / math.sqrt(F))
    choice = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)])
    pairs, max_tiles = T * top, ops.moe_max_tiles(T * top, E, tile)
    z = lambda n: torch.zeros(n, dtype=torch.int32, device="cuda")
    meta, tile_expert, slot_src, pair_slot = z(4), z(max_tiles), z(max_tiles * tile), z(pairs)
    ops.moe_group(choice.flatten().to(torch.int32).cuda(), pairs, E, meta, tile_expert, slot_src, pair_slot, max_tiles, tile)
    rows = torch.full((max_tiles * tile, W), float("nan"), device="cuda", dtype=torch.bfloat16)
    act = torch.full((max_tiles * tile, F), float("nan"), device="cuda", dtype=torch.bfloat16)
    y = torch.full((max_tiles * tile, W), float("nan"), device="cuda")
    ops.moe_gather(rows, dev(x, "bfloat16"), slot_src, meta, top, tile, max_tiles)
    ops.moe_gemm_tc(rows, tile_expert, meta, dev(up, "bfloat16"), act, max_tiles, act="relu2", tile=tile)
    ops.moe_gemm_tc(act, tile_expert, meta, dev(down, "bfloat16"), y, max_tiles, tile=tile)
    assert ops.gemm_tc_take_error() == 0
    a = torch.stack([P.relu_squared(x[t].double() @ up[int(e)].double().T) for t in range(T) for e in choice[t]])
    slots = pair_slot.cpu().long()
    assert max_err(act[slots.cuda()], a) < KTOL["bfloat16"]
    ref = torch.stack([bf(a[i].float()).double() @ down[int(e)].double().T for i, e in enumerate(choice.flatten())])
    assert max_err(y[slots.cuda()], ref) < 2e-2


def _lightning_inputs(T, H, D, V, seed):
    g = torch.Generator().manual_seed(seed)
    q, k, v = bf(torch.randn(T, H * D, generator=g)), bf(torch.randn(T, H * D, generator=g)), bf(torch.randn(T, H * V, generator=g))
    decay = ([0.0, 1.0, 0.6, 0.9, 0.99, 0.999] * 2)[seed % 3:][:H]
    return q, k, v, decay


def _plain_lightning(q, k, v, decay, H, D, V, activated=False):
    act = (lambda x: x) if activated else P.silu
    T = q.shape[0]
    o, S = P.lightning_recurrence(act(q.double()).view(T, H, D), act(k.double()).view(T, H, D), act(v.double()).view(T, H, V), decay)
    return o.reshape(T, H * V), S


LIGHTNING_SIZES = [(1, 16, 8), (2, 16, 24), (3, 10, 6), (2, 48, 64), (5, 64, 32), (1, 100, 130), (2, 256, 8), (4, 128, 128), (2, 32, 200)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,V", LIGHTNING_SIZES)
def test_fixed_decay_recurrence_in_steps_equals_the_plain_loop(dtype, H, D, V):
    """Token by token in portions through other slots, beside a single token of another request, as segments of a long step,
    and (sizes that it takes) with the single-token kernel in between."""
    from llm_b200.csrc import ops
    T = 300
    q, k, v, decay = _lightning_inputs(T, H, D, V, H * 1000 + D)
    ref, S_ref = _plain_lightning(q, k, v, decay, H, D, V)
    proj, dec = dev(torch.cat([q, k, v], dim=1), dtype), dev(torch.tensor(decay))
    cols = lambda p: (p[:, :H * D], p[:, H * D:2 * H * D], p[:, 2 * H * D:])
    scale = float(ref.abs().max())
    state = torch.zeros(4, H * D * V, device="cuda")
    out = torch.empty(T, H * V, device="cuda")
    at = 0
    for n in (40, 1, 2, 17, 1, 64, 5, 1, 1, 100, 68):
        # the request in slot 2, a single token of another request (slot 0) in front of it
        rows = torch.cat([proj[:1], proj[at:at + n]]).contiguous()
        o = torch.empty(1 + n, H * V, device="cuda")
        ctx = step_ctx([1, n], [0, 2])
        if n == 1 and ops.lightning_decode_available(D, V, state):
            ops.lightning_decode(o, rows, dec, state, ctx, H, D, V)
        else:
            ops.const_scan(o, *cols(rows), dec, state, ctx, H, D, V)
        out[at:at + n] = o[1:]
        at += n
    assert at == T and max_err(out, ref) < 2e-5 and max_err(state[2], S_ref.flatten()) < 2e-5
    assert float(state[1].abs().max()) == 0 and float(state[3].abs().max()) == 0
    state.zero_()
    seg_state, seg_decay = torch.zeros((T // 64 + 1) * H * D * V, device="cuda"), torch.zeros((T // 64 + 1) * H * D, device="cuda")
    ops.const_scan(out, *cols(proj), dec, state, step_ctx([T], [1]), H, D, V, seg_len=64, seg_state=seg_state, seg_decay=seg_decay)
    assert max_err(out, ref) < 2e-5 and max_err(state[1], S_ref.flatten()) < 2e-5 and scale > 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,V", [(2, 16, 24), (3, 10, 8), (4, 128, 128), (1, 512, 12), (2, 200, 68)])
def test_single_token_kernel_sums_partial_results(dtype, H, D, V):
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(D)
    B = 5
    proj = torch.randn(B, H * (2 * D + V), generator=g)
    S0, decay = torch.randn(7, H, D, V, generator=g), [0.9, 0.0, 1.0, 0.5][:H]
    slots = [6, 0, 3, 1, 5]
    buf, make = partials_of(proj, 4, g)
    state, out = dev(S0.view(7, -1)), torch.empty(B, H * V, device="cuda")
    ops.lightning_decode(out, make(buf, DT[dtype]), dev(torch.tensor(decay)), state, step_ctx([1] * B, slots), H, D, V)
    a = P.silu(proj.double())
    for e, s in enumerate(slots):
        o, S = P.lightning_recurrence(a[e:e + 1, :H * D].view(1, H, D), a[e:e + 1, H * D:2 * H * D].view(1, H, D),
                                      a[e:e + 1, 2 * H * D:].view(1, H, V), decay, S0[s].double())
        assert max_err(out[e], o.flatten()) < 2e-5 and max_err(state[s], S.flatten()) < 2e-6
    for s in (2, 4):
        assert torch.equal(state[s].cpu(), S0[s].flatten())


@pytest.mark.parametrize("H,D,V", [(1, 16, 8), (2, 16, 24), (3, 48, 40), (2, 64, 64), (4, 128, 128), (1, 256, 8), (2, 32, 200), (6, 32, 72)])
def test_chunk_wise_form_equals_the_plain_loop(H, D, V):
    """A step of five entries (one token, a chunk exactly, one more than two chunks, a portion off every border, a long one)
    from non-zero states.  The factors are bfloat16; everything else carries float32's accuracy."""
    from llm_b200.csrc import ops
    lens, T0 = [1, 64, 129, 77, 300], 30
    seqs = [_lightning_inputs(T0 + n, H, D, V, 100 * H + D) for n in lens]
    decay = seqs[0][3]
    dec = dev(torch.tensor(decay))
    state = torch.zeros(6, H * D * V, device="cuda")
    refs, starts = [], []
    for q, k, v, _ in seqs:
        o, S = _plain_lightning(q, k, v, decay, H, D, V, activated=True)
        _, S0 = _plain_lightning(q[:T0], k[:T0], v[:T0], decay, H, D, V, activated=True)
        refs.append((o[T0:], S))
        starts.append(S0)
    slots = [5, 2, 0, 4, 1]
    for s, S0 in zip(slots, starts):
        state[s] = dev(S0.flatten())
    qkv = torch.cat([torch.cat([q[T0:], k[T0:], v[T0:]], dim=1) for q, k, v, _ in seqs])
    qkv = dev(qkv, "bfloat16")
    T = sum(lens)
    out = torch.full((T, H * V), float("nan"), device="cuda")
    scratch = torch.full((ops.lightning_chunk_scratch(T // 64 + len(lens), H, D, V),), float("nan"), device="cuda")
    ops.lightning_chunks(out, qkv[:, :H * D], qkv[:, H * D:2 * H * D], qkv[:, 2 * H * D:], dec, state, step_ctx(lens, slots), H, D, V, scratch)
    at = 0
    for (o, S), s, n in zip(refs, slots, lens):
        assert max_err(out[at:at + n], o) < 4e-6 and max_err(state[s], S.flatten()) < 4e-6
        at += n
    assert float(state[3].abs().max()) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,R,C,width", [(3, 16, 8, 24, 32), (2, 10, 6, 22, 28), (8, 64, 32, 96, 128), (1, 9, 2, 11, 64), (4, 128, 64, 512, 576),
                                           (2, 8, 0, 16, 16)])
def test_queries_and_cache_rows_of_one_product(dtype, H, D, R, C, width):
    """Queries turned, the latent normed, the shared key part turned, both with the factor on cos and sin; rows in shuffled
    places, padded with zeros; from a tensor and from partial results; and the queries of a layer without latents."""
    from llm_b200.csrc import ops
    g = torch.Generator().manual_seed(H * 100 + D)
    T, page, eps, amp = 7, 16, 1e-5, 1.37
    per = H * (R + D)
    x = torch.randn(T, per + C + R, generator=g)
    gain = torch.randn(C, generator=g)
    positions = [0, 1, 5, 90, 700, 3000, 16]
    slots = [3, 40, 17, 0, 63, 32, 31]
    freqs = torch.rand(R // 2, generator=g) * 0.5
    half = lambda t: torch.cat([t[..., 0:R:2], t[..., 1:R:2]], dim=-1)             # neighbours -> rotate-half order
    back = lambda t: torch.stack([t[..., :R // 2], t[..., R // 2:]], dim=-1).flatten(-2)
    ang = (torch.tensor(positions).float().unsqueeze(1) * freqs).double()          # the angle is one float32 product
    turn = lambda t: back(P.rotate_halves(half(t.double()), torch.ones(T), [1.0] * (R // 2), amp, ang)) if R else t.double()
    q = x[:, :per].view(T, H, R + D)
    q_ref = torch.cat([torch.stack([turn(q[:, h, :R]) for h in range(H)], dim=1), q[:, :, R:].double()], dim=-1).reshape(T, per)
    row_ref = torch.cat([turn(x[:, per + C:]), P.rms_norm(x[:, per:per + C].double(), gain.double(), eps),
                         torch.zeros(T, width - R - C, dtype=torch.float64)], dim=-1)
    buf, make = partials_of(x, 3, g)
    tol = 2e-6 if dtype == "float32" else KTOL["bfloat16"]
    fd = dev(freqs) if R else None
    for term in (dev(x), make(buf, torch.float32)):
        pages = torch.full((4, 1, page, width), 7.0, device="cuda", dtype=DT[dtype])
        out = torch.empty(T, per, device="cuda", dtype=DT[dtype])
        ops.latent_q_rope_store(term, out, H, D, dev(gain), C, R, fd, amp, i32(positions), eps, i32(slots), pages, T)
        flat = pages.view(-1, width)
        assert max_err(out, q_ref) < 4 * tol and max_err(flat[slots], row_ref) < 4 * tol
        untouched = [s for s in range(64) if s not in slots]
        assert float(flat[untouched].float().min()) == 7.0
    out.zero_()
    ops.latent_q_rope_store(dev(x), out, H, D, None, 0, R, fd, amp, i32(positions), eps, None, None, T)
    assert max_err(out, q_ref) < 4 * tol


# ---- whole models ---------------------------------------------------------------------
LENGTHS = {"A": [1, 5, 33, 70, 129], "B": [2, 47, 64, 150, 330], "C": [3, 40, 17, 90], "D": [1, 16, 31, 100], "E": [1, 260, 31, 193],
           "F": [2, 33, 140, 95], "G": [1, 2, 60, 257]}
MARGIN = 0.03      # bfloat16: a choice of experts (or of groups) that hangs on less than this may fall otherwise


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

    def get(name, decided=False):
        if (name, decided) not in cache:
            cfg, page = CONFIGS[name]
            w = make_weights(cfg, seed=ord(name), decided=decided)
            reqs = {f"r{i}": random_tokens(n, cfg["vocab"], 300 + i) for i, n in enumerate(LENGTHS[name])}
            ref = {rid: plain(cfg, w, toks) for rid, toks in reqs.items()}
            upto = {rid: clear_rows(cfg, w, toks) for rid, toks in reqs.items()}
            cache[name, decided] = (cfg, page, w, reqs, ref, upto)
        return cache[name, decided]
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


# "decided": bfloat16 with routers whose choices no rounding moves, so that every row is compared
MODES = ["float32", "bfloat16", "decided"]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_cut_matches_plain(models, name, mode):
    dtype = "bfloat16" if mode == "decided" else mode
    cfg, page, w, reqs, ref, upto = models(name, mode == "decided")
    assert mode != "decided" or all(upto[rid] == len(toks) for rid, toks in reqs.items())
    longest = max(len(t) for t in reqs.values())
    eng = make_engine(cfg, w, dtype, page, -(-longest // page) + 1)       # a pool barely larger than the longest request
    compare(replay.run_steps(eng, replay.steps_whole(reqs)), ref, dtype, "whole", upto)
    compare(replay.run_steps(eng, replay.steps_tail_decode(reqs)), ref, dtype, "tail decode", upto)
    compare(replay.run_steps(eng, replay.steps_portions(reqs)), ref, dtype, "portions", upto)
    compare(replay.run_steps(eng, replay.steps_portions(reqs, sizes=(2, 2, 3, 2, 16, 2, 17, 64))), ref, dtype, "small portions", upto)
    compare(replay.run_steps(eng, replay.steps_portions(reqs, sizes=(195, 63, 2, 70))), ref, dtype, "large portions", upto)
    eng.check_status()
    eng.cache.check()
    assert all(eng.cache.num_free_pages(g) == eng.cache.group_spec(g).num_pages for g in range(eng.cache.num_groups))
    lens = sorted((len(t) for t in reqs.values()), reverse=True)
    eng = make_engine(cfg, w, dtype, page, sum(-(-n // page) for n in lens[:4]) + 1)
    compare(replay.run_steps(eng, replay.steps_mixed(reqs)), ref, dtype, "mixed", upto)     # freed pages and slots are used again
    compare(replay.run_steps(eng, replay.steps_mixed(reqs, prefill_sizes=(200, 2, 130, 65))), ref, dtype, "mixed, long portions", upto)
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "G"])
def test_batch_of_unequal_requests_equals_each_alone(models, name, dtype):
    from llm_b200.engine.engine import StepEntry
    cfg, page, w, reqs, ref, upto = models(name, dtype == "bfloat16")
    eng = make_engine(cfg, w, dtype, page, 60)
    alone = replay.run_steps(eng, replay.steps_whole(reqs))
    entries = [StepEntry(rid, toks, list(range(len(toks)))) for rid, toks in reqs.items()][-4:]
    if sum(len(e.tokens) for e in entries) > 512:
        entries = entries[:-1]
    rows = eng.step(entries).float().cpu()
    at = 0
    for e in entries:
        n = len(e.tokens)
        m = n if dtype == "float32" else upto[e.request_id]
        if m:
            err = (rows[at:at + m] - alone[e.request_id][:m]).abs().max(dim=1).values / alone[e.request_id].abs().max()
            if dtype == "float32":
                assert float(err.max()) < 1e-5
            else:            # products of other row counts round differently: two bfloat16 results, each off the true one
                assert float(err.max()) < 1e-1 and float(err.median()) < 2e-2
        at += n
        eng.release(e.request_id)


NEEDLE, QUERY = 7, 11


def _far_key_model(borrowed: bool):
    """A latent attention (or one that borrows the latents of a layer before it that writes next to nothing) whose first head
    sends the token QUERY to the token NEEDLE: its unrotated query map gets a term that turns QUERY's row into NEEDLE's key."""
    own = latent(2, 32, 8, 16, 40, 0.2, 1e4, yarn(16.0, 128))
    layers = [layer(own, None)]
    if borrowed:
        layers.append(layer(latent(2, 32, 8, 16, 40, 0.2, 1e4, yarn(16.0, 128), kv_from=0), None))
    cfg = config(64, 80, 0.5, layers)
    w = make_weights(cfg, seed=11, peak=0.5)
    i = len(layers) - 1
    x = w["embed"].double()
    kept = P.latents(x[NEEDLE:NEEDLE + 1], {k: v.double() for k, v in P.sub(w, "l0.mix").items()}, own["mixer"], cfg["norm"]["eps"])
    if borrowed:              # the first layer leaves the stream as its own norm of the embedding
        w["l0.mix.o"] = w["l0.mix.o"] * 0.0
        x = P.centred_norm(cfg["postln_alpha"] * x, w["l0.norm1"].double(), cfg["norm"]["eps"])
    key = (kept[0] @ w[f"l{i}.mix.uk"].double()[:32].T)[0]
    row = x[QUERY]
    q = w[f"l{i}.mix.q"].double()
    q[:32] += torch.outer(key, row) * (20.0 / (0.2 * float(key @ key)) / float(row @ row))
    w[f"l{i}.mix.q"] = bf(q.float())
    return cfg, w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("borrowed", [False, True])
@pytest.mark.parametrize("place", [0, 5, 15, 16, 300])
def test_attention_finds_a_key_hundreds_of_tokens_back(dtype, borrowed, place):
    """One NEEDLE (the first token, inside a page, at its edges, far on), QUERY tokens later; the rows of the queries change when
    the needle is exchanged (plain side), and those are the strict ones.  A query ahead of the needle must not see it."""
    cfg, w = _far_key_model(borrowed)
    T, asks = 700, [place + 1, 400, 699]
    toks = [t if t not in (NEEDLE, QUERY) else t + 20 for t in random_tokens(T, cfg["vocab"], 3)]
    toks[place] = NEEDLE
    early = [place - 1] if place else []
    for i in asks + early:
        toks[i] = QUERY
    other = list(toks)
    other[place] = 33
    ref, ref_other = plain(cfg, w, toks), plain(cfg, w, other)
    moved = (ref - ref_other).abs().max(dim=1).values / ref.abs().max()
    assert float(moved[asks].min()) > 0.1, "premise: the far rows hang on the exchanged token"
    assert not early or float(moved[early].max()) == 0, "premise: an earlier row does not"
    tol, strict = (None if dtype == "float32" else 4e-2), asks + early
    eng = make_engine(cfg, w, dtype, 16, -(-T // 16) + 1, max_tokens=704)
    compare(replay.run_steps(eng, replay.steps_whole({"x": toks})), {"x": ref}, dtype, "whole", strict=strict, tol=tol)
    compare(replay.run_steps(eng, replay.steps_tail_decode({"x": toks}, tail=320)), {"x": ref}, dtype, "decode", strict=strict, tol=tol)
    compare(replay.run_steps(eng, replay.steps_portions({"x": toks}, sizes=(100, 2, 37, 128, 3)), ), {"x": ref}, dtype, "portions", strict=strict, tol=tol)
    compare(replay.run_steps(eng, replay.steps_whole({"y": other})), {"y": ref_other}, dtype, "exchanged", strict=strict, tol=tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_remembers_a_token_from_hundreds_back(dtype):
    """Slow decays; the request's state slot was another request's before; portions cut the sequence inside and at chunks."""
    cfg = config(48, 70, 0.5, [layer(lightning(2, 16, 24, [0.9999, 1.0]), None)])
    w = make_weights(cfg, seed=9)
    T, p = 700, 20
    toks = random_tokens(T, cfg["vocab"], 5)
    other = list(toks)
    other[p] = (toks[p] + 9) % cfg["vocab"]
    ref, ref_other = plain(cfg, w, toks), plain(cfg, w, other)
    moved = (ref - ref_other).abs().max(dim=1).values / ref.abs().max()
    assert float(moved[650:].max()) > 5e-4, "premise: the state still holds the exchanged token"      # float32 sees 3e-5
    eng = make_engine(cfg, w, dtype, 16, 50, max_tokens=512, max_seqs=2)
    replay.run_steps(eng, replay.steps_whole({"warm": random_tokens(90, cfg["vocab"], 1)}))      # uses and frees a slot
    for sizes in ((100, 2, 64, 1, 128, 31), (256, 192, 252), (193, 1, 1, 320, 2)):
        compare(replay.run_steps(eng, replay.steps_portions({"x": toks}, sizes=sizes)), {"x": ref}, dtype, f"portions {sizes}")
    compare(replay.run_steps(eng, replay.steps_portions({"y": other}, sizes=(128,))), {"y": ref_other}, dtype, "exchanged")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_slot_that_is_used_again_starts_from_zero(models, dtype):
    cfg, page, w, reqs, ref, upto = models("E")
    eng = make_engine(cfg, w, dtype, page, 40, max_seqs=1)           # one slot: every request takes the same one
    for _ in range(2):
        compare(replay.run_steps(eng, replay.steps_whole(reqs)), ref, dtype, "whole, one slot", upto)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "G"])
def test_long_decode_with_graphs_and_first_tokens(models, name, dtype):
    """One prompt token, then 210 decoded one by one under CUDA graphs, beside a second request that joins late."""
    cfg, page = CONFIGS[name]
    w = make_weights(cfg, seed=77, decided=dtype == "bfloat16")
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


def test_prefill_equals_token_by_token_from_the_first_token():
    for name in ("A", "E", "F"):
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
@pytest.mark.parametrize("seed", range(12))
def test_seeded_random_configurations(seed, dtype):
    cfg = random_config(seed)
    page = [8, 16, 32][seed % 3]
    w = make_weights(cfg, seed=1000 + seed, decided=dtype == "bfloat16")
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
@pytest.mark.parametrize("seed", range(6))
def test_seeded_configurations_of_layer_like_sizes(seed, dtype):
    cfg = random_config(100 + seed, large=True)
    w = make_weights(cfg, seed=2000 + seed, decided=dtype == "bfloat16")
    reqs = {f"r{i}": random_tokens(n, cfg["vocab"], seed * 10 + i) for i, n in enumerate([150, 40, 300])}
    ref = {rid: plain(cfg, w, toks) for rid, toks in reqs.items()}
    upto = {rid: clear_rows(cfg, w, toks) for rid, toks in reqs.items()}
    tol = 1e-4 if dtype == "float32" else 8e-2
    eng = make_engine(cfg, w, dtype, 16, 40)
    compare(replay.run_steps(eng, replay.steps_whole(reqs)), ref, dtype, f"seed {seed} whole", upto, tol=tol)
    compare(replay.run_steps(eng, replay.steps_mixed(reqs, prefill_sizes=(64, 2, 130, 200))), ref, dtype, f"seed {seed} mixed", upto, tol=tol)
    eng.check_status()
