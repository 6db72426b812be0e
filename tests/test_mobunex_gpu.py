"""Mobunex on the GPU against the plain implementation of tests/mobunex_oracle.py (float64): every mechanism alone, then the model
through the engine — whole prompts, token-by-token decoding, portions down to two tokens, long portions beside short ones, mixed
batches with reused pages and state slots, keys just inside and just outside every window, the first tokens of a sequence, long
decoding, other sizes and layer orders, greedy generation through the scheduler and the command line."""
import json
import math

import numpy as np
import pytest
import torch

import mobunex_oracle as mo

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
BF = torch.bfloat16
BOTH = [torch.float32, torch.bfloat16]


def _ops():
    from atoma_infer_b200 import hybrid_ops
    return hybrid_ops


@pytest.fixture(autouse=True)
def _reset_flags():
    yield
    if torch.cuda.is_available():
        _ops().debug_flags(0)


def nerr(got, want):
    got, want = torch.as_tensor(got).double().cpu(), torch.as_tensor(want).double().cpu()
    return float(((got - want) ** 2).mean().sqrt() / (want ** 2).mean().sqrt().clamp_min(1e-30))


def tol(dtype, f32=1e-5, bf16=2e-2):
    return f32 if dtype == torch.float32 else bf16


def bf(t):
    return t.to(BF).float()


def rnd(g, *shape, scale=1.0, shift=0.0):
    return bf(torch.randn(*shape, generator=g) * scale + shift)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def batch_layout(counts):
    """token_seq, query_start for sequences with `counts` tokens each in the step."""
    seq = [b for b, n in enumerate(counts) for _ in range(n)]
    return i32(seq), i32([0] + list(np.cumsum(counts)))


def paged(n_tokens, bs, g, extra=3):
    """Shuffled pages for sequences of n_tokens[b] tokens: block tables [B, max], per-token cache rows, rows of the pool."""
    need = [-(-n // bs) for n in n_tokens]
    perm = torch.randperm(sum(need) + extra, generator=g).tolist()
    tables, at = [], 0
    for k in need:
        tables.append(perm[at:at + k])
        at += k
    mb = max(need)
    bt = torch.tensor([t + [0] * (mb - len(t)) for t in tables], dtype=torch.int32)
    rows = [[tables[b][p // bs] * bs + p % bs for p in range(n)] for b, n in enumerate(n_tokens)]
    return bt, rows, (sum(need) + extra) * bs


# ------------------------------------------------------------------------------------------------
# the residual stream
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("W,depth,with_y", [(40, 0, True), (64, 1, True), (33, 2, True), (50, 5, True), (132, 9, True), (48, 1, False)])
def test_post_norm_update_and_average_over_depth(dtype, W, depth, with_y):
    """x <- norm(alpha x + y); the row joins the earlier ones and x becomes their weighted sum; rows behind it stay untouched."""
    g = torch.Generator().manual_seed(W + depth)
    T, eps, alpha = 6, 1e-4, 1.7
    x, y, gain = rnd(g, T, W), rnd(g, T, W), 1.3
    rows, dw = torch.randn(depth + 2, T, W, generator=g), torch.randn(max(1, depth), generator=g)
    n = mo.post_norm(x.double(), y.double() if with_y else 0.0, alpha, gain, eps)
    xd, dev_rows = x.to(DEV).clone(), rows.to(DEV).clone()
    h, trace = _ops().postnorm_residual(xd, torch.full((W,), gain, device=DEV), alpha, eps, dtype, y=y.to(dtype).to(DEV) if with_y else None,
                                        depth=dev_rows if depth else None, depth_w=dw.to(DEV) if depth else None, depth_n=depth, want_trace=True)
    want = n
    if depth:
        want = mo.depth_average([rows[j].double() for j in range(depth - 1)] + [n], dw.double())
        assert nerr(dev_rows[depth - 1], n) < 1e-6
        keep = [j for j in range(depth + 2) if j != depth - 1]
        assert torch.equal(dev_rows[keep].cpu(), rows[keep])
    assert nerr(xd, want) < 2e-6 and torch.equal(xd, trace)
    assert nerr(h, want) < tol(dtype, 2e-6, 4e-3)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("W,T", [(48, 7), (64, 300)])
def test_post_norm_update_sums_the_experts_rows(dtype, W, T):
    """Router, routed experts, shared expert and the update that adds them, against the plain mixture; an expert nobody chooses."""
    g = torch.Generator().manual_seed(W + T)
    E, top, ff, sff, eps, alpha = 6, 3, 32, 24, 1e-5, 0.8
    router = dict(experts=E, top=top, groups=dict(count=3, keep=2))
    P = {"router": rnd(g, E, W, scale=W ** -0.5), "correction": rnd(g, E, scale=0.2)}
    P["correction"][4] = -40.0
    for k in [f"e{e}." for e in range(E)] + ["shared."]:
        n = sff if k == "shared." else ff
        P[k + "gate"], P[k + "up"], P[k + "down"] = (rnd(g, n, W, scale=W ** -0.5), rnd(g, n, W, scale=W ** -0.5), rnd(g, W, n, scale=n ** -0.5))
    h, x = rnd(g, T, W), rnd(g, T, W)
    dv = lambda t: t.to(dtype).to(DEV)
    hd = dv(h)
    idx, wgt = _ops().moe_route_grouped(hd, P["router"].to(DEV), P["correction"].to(DEV), top, 3, 2, score="sigmoid", group_top=2)
    assert int((idx == 4).sum()) == 0
    gu = torch.stack([torch.cat([P[f"e{e}.gate"], P[f"e{e}.up"]]) for e in range(E)])
    eo, pr, ws = _ops().moe_expert_rows(hd, idx, wgt, dv(gu), dv(torch.stack([P[f"e{e}.down"] for e in range(E)])), 0.0, 1.0, 0.0)
    y = _ops().linear(_ops().glu(_ops().linear(hd, dv(torch.cat([P["shared.gate"], P["shared.up"]]))), 0), dv(P["shared.down"]))
    xd = x.to(DEV).clone()
    _ops().postnorm_residual(xd, torch.full((W,), 0.9, device=DEV), alpha, eps, dtype, y=y, experts=(eo, pr, idx, ws))
    P64 = {k: v.double() for k, v in P.items()}
    ff_out = mo.moe_ff(h.double(), P64, "", dict(router=router, shared=dict(ff=sff)))
    assert nerr(xd, mo.post_norm(x.double(), ff_out, alpha, 0.9, eps)) < tol(dtype, 3e-6, 1e-2)
    del ws


# ------------------------------------------------------------------------------------------------
# router
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("E,top,count,keep", [(8, 3, 4, 3), (12, 4, 3, 2), (16, 2, 8, 1), (6, 6, 2, 2), (5, 2, 5, 3), (9, 4, 1, 1), (64, 6, 8, 4), (4, 2, 2, 1)])
def test_groups_are_ranked_by_their_two_best_choice_scores(dtype, E, top, count, keep):
    g = torch.Generator().manual_seed(E * 10 + top)
    T, W = 40, 36
    h, wr, corr = rnd(g, T, W), rnd(g, E, W, scale=0.2), rnd(g, E, scale=0.5, shift=-0.6)      # corrected scores of both signs
    idx, wgt = _ops().moe_route_grouped(h.to(dtype).to(DEV), wr.to(DEV), corr.to(DEV), top, count, keep, score="sigmoid", group_top=2)
    P = {"router": wr.double(), "correction": corr.double()}
    by_one = 0
    for t in range(T):
        want = mo.route(h[t].double(), P, "", dict(experts=E, top=top, groups=dict(count=count, keep=keep) if count > 1 else None))
        assert [e for e, _ in want] == idx[t].tolist()
        assert nerr(wgt[t], torch.tensor([w for _, w in want])) < 3e-6
    one, _ = _ops().moe_route_grouped(h.to(dtype).to(DEV), wr.to(DEV), corr.to(DEV), top, count, keep, score="sigmoid", group_top=1)
    by_one = int((one != idx).any(1).sum())
    assert by_one > 0 if (keep < count and E > count) else by_one == 0      # ranking by the single best score chooses differently


def test_the_second_best_choice_score_decides():
    """Group 0 holds the single best output, group 1 two good ones: the sum ranks group 1 first."""
    wr = torch.zeros(4, 4)
    corr = torch.tensor([0.9, -0.9, 0.3, 0.2])
    h = torch.ones(1, 4)
    idx, wgt = _ops().moe_route_grouped(h.to(DEV), wr.to(DEV), corr.to(DEV), 2, 2, 1, score="sigmoid", group_top=2)
    assert idx.tolist() == [[2, 3]] and torch.allclose(wgt.cpu(), torch.tensor([[0.5, 0.5]]))
    idx, _ = _ops().moe_route_grouped(h.to(DEV), wr.to(DEV), corr.to(DEV), 2, 2, 1, score="sigmoid", group_top=1)
    assert idx.tolist() == [[0, 1]]


# ------------------------------------------------------------------------------------------------
# recurrent block
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("taps,C", [(1, 40), (2, 64), (3, 33), (4, 72), (6, 24)])
def test_short_filter_with_biases_over_portions_of_any_size(dtype, taps, C):
    """The input's bias is part of the input (and so of what is carried), the filter's is not; before the start there is zero, not the
    bias.  Sequences cut into unequal portions down to one token, on state slots that hold garbage."""
    g = torch.Generator().manual_seed(taps * 100 + C)
    lens, cuts, slots = [23, 9, 14], [[1, 1, 5, 2, 14], [9], [3, 1, 1, 1, 8]], [4, 0, 2]
    xs = [rnd(g, n, C) for n in lens]
    w, ib, ob = rnd(g, C, taps, scale=0.5), rnd(g, C), rnd(g, C)
    want = [mo.causal_conv(x.double() + ib.double(), w.double(), ob.double()) for x in xs]
    for flags in ((0, 2) if dtype == BF else (0,)):
        _ops().debug_flags(flags)
        hist = torch.full((5, max(1, taps - 1) * C + 3), 77.0, device=DEV)
        done = [0, 0, 0]
        for step in range(5):
            members = [b for b in range(3) if step < len(cuts[b])]
            counts = [cuts[b][step] for b in members]
            x = torch.cat([xs[b][done[b]:done[b] + c] for b, c in zip(members, counts)]).to(dtype).to(DEV)
            tseq, qs = batch_layout(counts)
            o, _ = _ops().tap_filter(x, w.to(DEV), None, hist, i32([slots[b] for b in members]), tseq, qs, i32([done[b] for b in members]), False, 0,
                                     in_bias=ib.to(DEV), bias1=ob.to(DEV))
            at = 0
            for b, c in zip(members, counts):
                assert nerr(o[at:at + c], want[b][done[b]:done[b] + c]) < tol(dtype, 1e-6, 8e-3), (step, b)
                at += c
                done[b] += c


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("blocks,n", [(1, 64), (3, 20), (2, 80), (5, 8), (2, 256), (4, 7)])
@pytest.mark.parametrize("T", [1, 70])
def test_gates_of_the_linear_recurrent_unit(dtype, blocks, n, T):
    """Decays from far below one to one minus 1e-6: sqrt(1 - a^2) must not cancel."""
    g = torch.Generator().manual_seed(blocks * 100 + n + T)
    C = blocks * n
    u, wr, wi = rnd(g, T, C), rnd(g, blocks, n, n, scale=n ** -0.5), rnd(g, blocks, n, n, scale=n ** -0.5)
    br, bi, lam = rnd(g, C), rnd(g, C), torch.linspace(-16.0, 4.0, C)
    rate = -8.0 * mo.softplus(lam.double())
    dec, inp = _ops().lru_gates(u.to(dtype).to(DEV), torch.cat([wr, wi], 1).to(dtype).to(DEV), br.to(DEV), bi.to(DEV), rate.float().to(DEV), blocks)
    r = mo.sigma(mo.blockwise(u.double(), wr.double(), br.double().reshape(blocks, n)))
    i = mo.sigma(mo.blockwise(u.double(), wi.double(), bi.double().reshape(blocks, n)))
    log_a = rate * r
    want = torch.sqrt(-torch.expm1(2 * log_a)) * i * u.double()
    assert float((dec.double().cpu() - torch.exp(log_a)).abs().max()) < 2e-6     # bfloat16 operands are exact here; sums are float32
    rel = (inp.double().cpu() - want).abs() / want.abs().clamp_min(1e-6 * float(want.abs().max()))
    assert float(rel.max()) < 2e-4 and nerr(inp, want) < 3e-6


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("flags", [0, 4])
@pytest.mark.parametrize("C", [40, 129])
def test_linear_scan_over_portions(dtype, flags, C):
    """Portions that take the blocked scan (128 tokens and more) and the one in token order, on slots that hold garbage; a sequence that
    starts anew on a used slot."""
    _ops().debug_flags(flags)
    g = torch.Generator().manual_seed(C)
    lens, cuts, slots = [700, 12, 133], [[1, 300, 2, 397], [12], [130, 1, 2]], [3, 1, 0]
    dec = [torch.rand(n, C, generator=g) * 0.5 + 0.5 for n in lens]
    inp = [torch.randn(n, C, generator=g) for n in lens]
    gate, gb = [rnd(g, n, C) for n in lens], rnd(g, C)
    want = []
    for d, x, y in zip(dec, inp, gate):
        s, rows = torch.zeros(C, dtype=F64), []
        for t in range(d.shape[0]):
            s = d[t].double() * s + x[t].double()
            rows.append(s)
        want.append((torch.stack(rows) * mo.gelu_tanh(y.double() + gb.double()), s))
    state = torch.full((4, C + 5), 9.0, device=DEV)
    for _ in range(2):                       # twice: the second time the slots hold the first run's state
        done = [0, 0, 0]
        for step in range(4):
            members = [b for b in range(3) if step < len(cuts[b])]
            counts = [cuts[b][step] for b in members]
            cat = lambda xs: torch.cat([xs[b][done[b]:done[b] + c] for b, c in zip(members, counts)])
            _, qs = batch_layout(counts)
            out = _ops().linear_scan(cat(dec).to(DEV), cat(inp).to(DEV), cat(gate).to(dtype).to(DEV), gb.to(DEV), state, i32([slots[b] for b in members]), qs,
                                     i32([done[b] for b in members]), max(counts))
            at = 0
            for b, c in zip(members, counts):
                assert nerr(out[at:at + c], want[b][0][done[b]:done[b] + c]) < tol(dtype, 2e-6, 4e-3), (step, b)
                at += c
                done[b] += c
        for b in range(3):
            assert nerr(state[slots[b], :C], want[b][1]) < 2e-6
    assert bool((state[2] == 9.0).all()) and bool((state[:, C:] == 9.0).all())


def test_a_write_far_back_is_still_in_the_state():
    """Decay one, a single write at token 0: 600 tokens later it reads back exactly, in one portion, in portions and token by token."""
    C, n = 33, 600
    dec, inp = torch.ones(n, C), torch.zeros(n, C)
    inp[0] = torch.arange(1, C + 1).float()
    gate = torch.full((n, C), 30.0)          # gelu(30) = 30
    for cuts in ([n], [7, 250, 2] + [1] * 20 + [n - 279], [1] * 40 + [n - 40]):
        state, done = torch.full((1, C), 5.0, device=DEV), 0
        for c in cuts:
            sl = slice(done, done + c)
            last = _ops().linear_scan(dec[sl].to(DEV), inp[sl].to(DEV), gate[sl].to(DEV), None, state, i32([0]), i32([0, c]), i32([done]), c)
            done += c
        assert torch.equal(last[-1].cpu(), inp[0] * 30.0), cuts


# ------------------------------------------------------------------------------------------------
# windowed softmax attention with biases, unit norms and a factor per head
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,D,V,window", [(4, 2, 16, 24, 9), (6, 3, 64, 64, 40), (5, 1, 10, 6, 3), (8, 8, 32, 16, 0), (4, 1, 128, 128, 17)])
def test_grouped_attention_on_a_mixed_batch(dtype, H, G, D, V, window):
    """A continued portion, a whole prompt and a decoded token in one step on shuffled pages; padding columns between the parts."""
    ops = _ops()
    g = torch.Generator().manual_seed(H * 100 + D)
    bs, eps, scale = 8, 1e-3, 0.7
    lens, starts = [53, 21, 40], [30, 0, 39]
    q_off, k_off = 0, H * D + 8
    v_off = k_off + G * D + 3
    N = v_off + G * V + 5
    proj, bias, temp = [rnd(g, n, N) for n in lens], rnd(g, N), rnd(g, H, shift=1.0)
    bt, rows, n_rows = paged(lens, bs, g)
    kc, vc = torch.full((n_rows, G, D), 50.0, dtype=dtype, device=DEV), torch.full((n_rows, G, V), 50.0, dtype=dtype, device=DEV)

    def step(members, spans):
        x = torch.cat([proj[b][lo:hi] for b, (lo, hi) in zip(members, spans)]).to(dtype).to(DEV)
        pos = torch.tensor([p for lo, hi in spans for p in range(lo, hi)], dtype=torch.int64, device=DEV)
        slot = torch.tensor([rows[b][p] for b, (lo, hi) in zip(members, spans) for p in range(lo, hi)], dtype=torch.int64, device=DEV)
        q = ops.qkv_headnorm_rope_cache(x, q_off, k_off, v_off, None, None, None, None, False, pos, slot, kc, vc, H, G, D, V, eps, bias=bias.to(DEV),
                                        q_head_scale=temp.to(DEV), unit_norm=True)
        tseq, qs = batch_layout([hi - lo for lo, hi in spans])
        return ops.softmax_attention_paged(q, kc, vc, pos, tseq, bt[members].contiguous().to(DEV), H, G, D, V, bs, scale, window=window, query_start=qs)

    step([0, 2], [(0, starts[0]), (0, starts[2])])
    got = step([0, 1, 2], [(starts[0], lens[0]), (0, lens[1]), (starts[2], lens[2])])
    at = 0
    for b in range(3):
        p = (proj[b] + bias).double()
        n = lens[b]
        part = lambda off, heads, dim: p[:, off:off + heads * dim].reshape(n, heads, dim)
        qh, kh, vh = mo.unit_rms(part(q_off, H, D), eps), mo.unit_rms(part(k_off, G, D), eps), part(v_off, G, V)
        want = mo.windowed_softmax(lambda i, h, lo, hi: (kh[lo:hi, h // (H // G)] @ qh[i, h]) * scale * temp[h].double(),
                                   lambda h, lo, hi: vh[lo:hi, h // (H // G)], n, H, V, window).reshape(n, H * V)[starts[b]:]
        assert nerr(got[at:at + want.shape[0]], want) < tol(dtype, 1e-5, 2e-2), b
        at += want.shape[0]


# ------------------------------------------------------------------------------------------------
# latent attention
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims,base,scaling", [(24, 30000.0, dict(factor=6.0, original=2048, fast=24.0, slow=1.5)), (8, 500.0, dict(factor=3.0, original=64, fast=4.0, slow=2.0)),
                                               (64, 1e6, dict(factor=40.0, original=4096, fast=30.0, slow=1.0)), (2, 100.0, dict(factor=2.0, original=16, fast=1.0, slow=1.0)),
                                               (16, 10000.0, None)])
def test_yarn_frequencies_and_exact_angles(dims, base, scaling):
    """The description's frequencies against the plain rule, and a rotation at position 300 000 that float32 angles would miss by 1e-2."""
    from atoma_infer_b200.hybrid import RotarySpec
    f, amp = mo.yarn_frequencies(dims, base, scaling)
    r = RotarySpec(dims=dims, base=base, interleaved=True, yarn=None if scaling is None else tuple(scaling[k] for k in ("factor", "original", "fast", "slow")))
    assert abs(r.amplitude - amp) < 1e-15 and nerr(torch.tensor(r.frequencies(), dtype=F64), f) < 1e-14
    hi = f.float()
    lo = (f - hi.double()).float()
    g = torch.Generator().manual_seed(dims)
    H, n = 3, dims + 4
    x, pos = torch.randn(5, H * n, generator=g), torch.tensor([0, 1, 77, 4099, 300000])
    xd = x.to(DEV).clone()
    _ops().rotate_heads(xd, pos.to(DEV), hi.to(DEV), H, n, True, 1.0, freq_lo=lo.to(DEV), amplitude=amp)
    want = mo.rotate_pairs(x.double().reshape(5, H, n), pos, f, amp)
    assert float((xd.cpu().double().reshape(5, H, n) - want).abs().max()) < 2e-6 * max(1.0, amp) * 4


def latent_case(g, H, D, Rd, V, Rq, Rk, W, scaling=True):
    m = dict(heads=H, dim=D, rot_dim=Rd, vdim=V, q_rank=Rq, kv_rank=Rk, scale=1.3 / math.sqrt(D + Rd),
             rot=dict(base=700.0, dims=Rd, scaling=dict(factor=5.0, original=32, fast=6.0, slow=1.0) if scaling else None))
    P = {"dq": rnd(g, Rq, W, scale=0.3), "dq.norm": rnd(g, Rq, shift=1.0, scale=0.1), "uq": rnd(g, H * (D + Rd), Rq, scale=2.0 * Rq ** -0.5),
         "dkv": rnd(g, Rk + Rd, W, scale=0.4), "dkv.norm": rnd(g, Rk, shift=1.0, scale=0.1), "uk": rnd(g, H * D, Rk, scale=Rk ** -0.5),
         "uv": rnd(g, H * V, Rk, scale=Rk ** -0.5), "g": rnd(g, H * V, W, scale=0.4), "o": torch.eye(H * V)}
    return m, P


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,D,Rd,V,Rq,Rk,window", [(3, 16, 8, 16, 24, 32, 7), (7, 64, 64, 32, 72, 192, 20), (2, 10, 6, 12, 9, 14, 0), (4, 32, 64, 48, 40, 128, 33),
                                                  (5, 16, 64, 16, 24, 192, 11)])
def test_latent_attention_on_a_mixed_batch(dtype, H, D, Rd, V, Rq, Rk, window):
    ops = _ops()
    g = torch.Generator().manual_seed(H * 10 + Rd)
    bs, eps, W = 8, 1e-5, 24
    lens, starts = [45, 20, 33], [20, 0, 32]
    m, P = latent_case(g, H, D, Rd, V, Rq, Rk, W)
    if window:
        m["mask"] = dict(size=window)
    hs = [rnd(g, n, W) for n in lens]
    f, amp = mo.yarn_frequencies(Rd, 700.0, m["rot"]["scaling"])
    freq, freq_lo = f.float().to(DEV), (f - f.float().double()).float().to(DEV)
    bt, rows, n_rows = paged(lens, bs, g)
    cache = torch.full((n_rows, Rk + Rd), 30.0, dtype=dtype, device=DEV)
    w_in, w_g = torch.cat([P["dq"], P["dkv"]]).to(dtype).to(DEV), P["g"].to(dtype).to(DEV)

    def step(members, spans):
        h = torch.cat([hs[b][lo:hi] for b, (lo, hi) in zip(members, spans)]).to(dtype).to(DEV)
        pos = torch.tensor([p for lo, hi in spans for p in range(lo, hi)], dtype=torch.int64, device=DEV)
        slot = torch.tensor([rows[b][p] for b, (lo, hi) in zip(members, spans) for p in range(lo, hi)], dtype=torch.int64, device=DEV)
        proj = ops.linear(h, w_in)
        cq = ops.latent_norm_rope_cache(proj, P["dq.norm"].to(DEV), P["dkv.norm"].to(DEV), freq, True, pos, slot, cache, Rq, Rk, Rd, eps, freq_lo=freq_lo,
                                        amplitude=amp)
        q = ops.linear(cq, P["uq"].to(dtype).to(DEV))
        qlat = ops.latent_query_absorb_rope(q, P["uk"].to(dtype).to(DEV), freq, True, pos, H, D, Rd, Rk, freq_lo=freq_lo, amplitude=amp)
        tseq, qs = batch_layout([hi - lo for lo, hi in spans])
        olat = ops.latent_attention_paged(qlat.reshape(qlat.shape[0], -1), cache, pos, tseq, bt[members].contiguous().to(DEV), None, H, Rk + Rd, bs, window,
                                          m["scale"], max(hi - lo for lo, hi in spans), query_start=qs, out_cols=Rk)
        return ops.latent_expand_values(olat.reshape(-1, H, Rk + Rd), P["uv"].to(dtype).to(DEV), H, V, Rk, dtype, gate=ops.linear(h, w_g))

    step([0, 2], [(0, starts[0]), (0, starts[2])])
    got = step([0, 1, 2], [(starts[0], lens[0]), (0, lens[1]), (starts[2], lens[2])])
    P64 = {k: v.double() for k, v in P.items()}
    at = 0
    for b in range(3):
        want = mo.latent_attention(hs[b].double(), P64, "", m, eps, list(range(lens[b])))[starts[b]:]
        assert nerr(got[at:at + want.shape[0]], want) < tol(dtype, 2e-5, 3e-2), b
        at += want.shape[0]


@pytest.mark.parametrize("H,D,Rd,V,Rk,window", [(4, 64, 24, 64, 96, 100), (2, 128, 64, 128, 192, 0), (3, 128, 64, 128, 512, 150), (2, 48, 16, 64, 64, 33),
                                                (2, 96, 32, 128, 64, 300), (2, 64, 64, 64, 64, 1), (1, 128, 56, 128, 72, 129)])
def test_long_portions_on_whole_keys(H, D, Rd, V, Rk, window):
    """Sequences with at least 128 tokens in the step: cached rows gathered from the pages, whole keys (plain and rotated part) and values
    expanded, windowed softmax on the tensor-memory kernel with keys longer than values, the gate on its outputs; the other
    sequences' rows are left alone."""
    ops = _ops()
    g = torch.Generator().manual_seed(H * 100 + Rd)
    seqs, bs = [(0, 300), (37, 1), (200, 150), (16, 2), (500, 128), (3, 257)], 16
    lens = [c + n for c, n in seqs]
    bt, rows, n_rows = paged(lens, bs, g)
    cache = torch.full((n_rows, Rk + Rd), 40.0, dtype=BF, device=DEV)
    lat = [rnd(g, n, Rk + Rd) for n in lens]
    for b in range(len(seqs)):
        cache[torch.tensor(rows[b], device=DEV)] = lat[b].to(BF).to(DEV)
    wk, wv = rnd(g, H * D, Rk, scale=Rk ** -0.5), rnd(g, H * V, Rk, scale=Rk ** -0.5)
    whole = torch.zeros(H, D + Rd, Rk + Rd)
    whole[:, :D, :Rk], whole[:, D:, Rk:] = wk.reshape(H, D, Rk), torch.eye(Rd)
    T = sum(n for _, n in seqs)
    q, gate = rnd(g, T, H * (D + Rd)), rnd(g, T, H * V + 8)
    scale = 1.5 / math.sqrt(D + Rd)
    _, qs = batch_layout([n for _, n in seqs])
    long_ = [(c, n) for c, n in seqs if n >= 128]
    max_keys = sum(n + (min(c, window - 1) if window else c) for c, n in long_)
    out = torch.full((T, H * V), 7.0, dtype=BF, device=DEV)
    dv = lambda t: t.to(BF).to(DEV)
    ops.latent_attention_expanded(dv(q), cache, dv(whole.reshape(H * (D + Rd), -1)), dv(wv), qs, i32([c for c, _ in seqs]), bt.to(DEV), None, H, D, Rk, bs, window,
                                  scale, 128, max(n for _, n in seqs), max(lens), max_keys, out=out, rot_dim=Rd, vdim=V, gate=dv(gate))
    at = 0
    for b, (c, n) in enumerate(seqs):
        got = out[at:at + n]
        if n < 128:
            assert bool((got == 7.0).all()), b
        else:
            k = torch.cat([(lat[b][:, :Rk].double() @ wk.double().T).reshape(-1, H, D), lat[b][:, None, Rk:].double().expand(-1, H, Rd)], 2)
            v = (lat[b][:, :Rk].double() @ wv.double().T).reshape(-1, H, V)
            sc = torch.einsum("ihd,jhd->hij", q[at:at + n].double().reshape(n, H, D + Rd), k) * scale
            dist = torch.arange(c, c + n)[:, None] - torch.arange(c + n)[None, :]
            sc = sc.masked_fill((dist < 0) | ((dist >= window) if window else (dist < 0)), -math.inf)
            want = torch.einsum("hij,jhv->ihv", torch.softmax(sc, -1), v).reshape(n, H * V) * mo.sigma(gate[at:at + n, :H * V].double())
            assert nerr(got, want) < 1.5e-2, b
        at += n
    assert ops.prefill_timeouts() == 0


@pytest.mark.parametrize("kind", ["latent", "latent_long", "softmax", "softmax_long"])
@pytest.mark.parametrize("far", [1, 15, 16, 17, 63, 64, 200, 511])
def test_one_loud_key_at_the_edge_of_the_window(kind, far):
    """One key's score stands far above the rest.  A query `far` tokens later reads (only) that key's value through a window of far + 1
    tokens and nothing of it through a window of far tokens — decoded alone, in a short portion and in a long one."""
    ops = _ops()
    g = torch.Generator().manual_seed(far)
    long_, D, bs = kind.endswith("long"), 64, 16
    dtype = BF
    before = 40                                          # tokens ahead of the loud key
    n = before + far + 1
    portions = [max(150, far + 2)] if long_ else [1, 2]
    for count in portions:
        if count > n:
            before, n = before + count - n, count
        loud, start = before, n - count
        bt, rows, n_rows = paged([n], bs, g)
        idx = torch.tensor(rows[0], device=DEV)
        k, v = rnd(g, n, D, scale=0.01), rnd(g, n, D)
        k[loud] = 0
        k[loud, 0] = 16.0
        q = torch.zeros(count, D)
        q[-1, 0] = 16.0
        pos, qs = torch.arange(start, n, device=DEV), i32([0, count])
        for window, seen in ((far + 1, True), (far, False)):
            if kind.startswith("softmax"):
                kc, vc = (torch.zeros((n_rows, 1, D), dtype=dtype, device=DEV) for _ in range(2))
                kc[idx, 0], vc[idx, 0] = k.to(dtype).to(DEV), v.to(dtype).to(DEV)
                out = ops.softmax_attention_paged(q.to(dtype).to(DEV), kc, vc, pos, i32([0] * count), bt.to(DEV), 1, 1, D, D, bs, 1.0, window=window,
                                                  query_start=qs, long_min_q=128 if long_ else 0)
            else:
                cache = torch.zeros((n_rows, D), dtype=dtype, device=DEV)
                both = k.clone()
                both[:, 1:] = v[:, 1:]                   # keys = values = the row: column 0 makes the score
                cache[idx] = both.to(dtype).to(DEV)
                v = both
                if long_:
                    eye = torch.eye(D).to(dtype).to(DEV)
                    out = ops.latent_attention_expanded(q.to(dtype).to(DEV), cache, eye, eye, qs, i32([start]), bt.to(DEV), None, 1, D, D, bs, window, 1.0, 128,
                                                        count, n, n)
                else:
                    out = ops.latent_attention_paged(q.to(DEV), cache, pos, i32([0] * count), bt.to(DEV), None, 1, D, bs, window, 1.0, count, query_start=qs)
            got = out.reshape(count, D)[-1].double().cpu()
            lo = max(0, n - 1 - window + 1)
            want = torch.softmax(k[lo:, 0].double() * 16.0, 0) @ v[lo:].double()
            assert float((got - want).abs().max()) < 3e-2
            close = float((got[1:] - v[loud, 1:].double()).abs().max()) < 3e-2
            assert close == seen, (count, window)


# ------------------------------------------------------------------------------------------------
# the model through the engine
# ------------------------------------------------------------------------------------------------
def make_engine(tmp_path, cfg, weights, dtype, max_tokens=512, block_size=16, live=4, budget=2048):
    from atoma_infer_b200 import checkpoint
    from atoma_infer_b200.engine import Engine
    tmp_path.mkdir(exist_ok=True)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    checkpoint.write_safetensors(tmp_path / "model.safetensors", {k: v.to(BF) for k, v in weights.items()})
    return Engine.from_model_dir(tmp_path, dtype=dtype, device=DEV, max_tokens=max_tokens, block_size=block_size,
                                 max_live_requests=live, max_num_batched_tokens=budget)


VARIANTS = {
    "base": dict(),
    "other_order": dict(kinds=("rglru", "latent_attention", "attention", "rglru", "attention"), mlps=("dense", None, None, "dense", "moe"), alpha=0.7, eps=1e-3),
    "plain": dict(kinds=("latent_attention", "attention"), mlps=("moe", "dense"), router=dict(experts=5, top=2, groups=None), shared_ff=0,
                  attention=dict(mask=None), latent=dict(mask=None, rot=dict(base=800.0, dims=8))),
    "odd_sizes": dict(width=50, vocab=37, ff=22, alpha=4.0, kinds=("rglru", "attention", "latent_attention", "rglru"), mlps=("dense", "moe", "moe", "moe"),
                      attention=dict(heads=6, kv_heads=3, dim=12, vdim=10, scale=0.4, mask=dict(size=5)),
                      latent=dict(heads=5, dim=12, rot_dim=6, vdim=10, q_rank=20, kv_rank=18, scale=0.3, mask=dict(size=70),
                                  rot=dict(base=777.0, dims=6, scaling=dict(factor=2.0, original=50, fast=3.0, slow=1.0))),
                      rglru=dict(width=35, blocks=5, conv=3), router=dict(experts=9, top=4, groups=dict(count=3, keep=1)), expert_ff=14, shared_ff=10),
    "one_of_each": dict(kinds=("attention", "rglru", "latent_attention"), attention=dict(heads=1, kv_heads=1, dim=16, vdim=16, mask=dict(size=1)),
                        latent=dict(heads=1, mask=dict(size=2)), rglru=dict(width=24, blocks=1, conv=1), router=dict(experts=4, top=1, groups=dict(count=4, keep=2))),
    "heads_of_64": dict(width=64, kinds=("attention", "latent_attention", "rglru"),
                        attention=dict(heads=4, kv_heads=1, dim=64, vdim=64, scale=0.125, mask=dict(size=50)),
                        latent=dict(heads=2, dim=64, rot_dim=40, vdim=64, q_rank=48, kv_rank=96, scale=0.1, mask=dict(size=200)),
                        rglru=dict(width=128, blocks=2, conv=2)),
    "heads_of_128": dict(width=64, kinds=("latent_attention", "attention"), mlps=("dense", "dense"),
                         attention=dict(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.09, mask=dict(size=300)),
                         latent=dict(heads=2, dim=128, rot_dim=64, vdim=128, q_rank=40, kv_rank=64, scale=0.07, mask=dict(size=140),
                                     rot=dict(base=1e5, dims=64, scaling=dict(factor=10.0, original=256, fast=16.0, slow=1.0)))),
}


def build(name, seed=0):
    g = torch.Generator().manual_seed(700 + seed)
    cfg = mo.random_config(**VARIANTS[name])
    return cfg, mo.random_weights(cfg, g), g


def median_row_error(got, want):
    """The typical row: in bfloat16 a near-tie of the router's choice legitimately takes another expert."""
    got, want = torch.as_tensor(got).double().cpu(), torch.as_tensor(want).double().cpu()
    e = ((got - want) ** 2).mean(-1).sqrt() / (want ** 2).mean().sqrt()
    return float(e.median())


def matches(got, want, dtype, f32=1e-5, bf16=4e-2):
    return nerr(got, want) < f32 if dtype == torch.float32 else median_row_error(got, want) < bf16


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", list(VARIANTS))
def test_whole_prompt_matches_the_plain_model(tmp_path, dtype, name):
    cfg, w, g = build(name)
    toks = torch.randint(0, cfg["vocab"], (83,), generator=g).tolist()
    want, layers = mo.forward(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, dtype)
    out = eng.step_forced([("a", toks, list(range(len(toks))))], want_residual_trace=True)
    assert out.residual_trace.shape[0] == len(layers)
    for i in range(len(layers)):
        assert matches(out.residual_trace[i], layers[i], dtype, 5e-6, 3e-2), i
    assert matches(out.logits, want, dtype)


@pytest.mark.parametrize("name", list(VARIANTS))
def test_decoding_token_by_token_equals_the_whole_prompt(tmp_path, name):
    """90 single-token steps on pages of four tokens: every page border, the first tokens of the sequence (where the filter still looks
    before its start), windows that fill up and then slide."""
    cfg, w, g = build(name, 1)
    toks = torch.randint(0, cfg["vocab"], (90,), generator=g).tolist()
    want, _ = mo.forward(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, torch.float32, max_tokens=128, block_size=4)
    got = [eng.step_forced([("a", [t], [0])]).logits.clone() for t in toks]
    assert nerr(torch.cat(got), want) < 1e-5


def test_long_decoding(tmp_path):
    """A short prompt and 400 decoded tokens: the state is carried for hundreds of steps, the windows slide over many pages."""
    cfg, w, g = build("base", 2)
    toks = torch.randint(0, cfg["vocab"], (420,), generator=g).tolist()
    want, _ = mo.forward(cfg, w, toks)
    for dtype in BOTH:
        eng = make_engine(tmp_path, cfg, w, dtype, max_tokens=512, block_size=16)
        eng.step_forced([("a", toks[:20], [])])
        got = [eng.step_forced([("a", [t], [0])]).logits.clone() for t in toks[20:]]
        assert matches(torch.cat(got), want[20:], dtype, 2e-5, 5e-2)
        eng.finish_request("a")


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["base", "other_order", "odd_sizes", "heads_of_64"])
@pytest.mark.parametrize("sizes", [[2, 2, 2, 3, 2], [40, 2, 17, 1, 1, 2, 64, 5], [1, 130, 1, 1], [19, 20, 21]])
def test_portions_of_any_size_equal_the_whole_prompt(tmp_path, dtype, name, sizes):
    cfg, w, g = build(name, 3)
    toks = torch.randint(0, cfg["vocab"], (sum(sizes),), generator=g).tolist()
    want, _ = mo.forward(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, dtype, max_tokens=256, block_size=8)
    got, at = [], 0
    for n in sizes:
        got.append(eng.step_forced([("a", toks[at:at + n], list(range(n)))]).logits.clone())
        at += n
    assert matches(torch.cat(got), want, dtype)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["heads_of_64", "heads_of_128", "base"])
def test_long_portions_beside_short_ones_and_decoded_tokens(tmp_path, dtype, name):
    """Portions of 128 tokens and more (bfloat16 heads of 64 / 128: tensor-memory kernels; the blocked scan) in one step with short
    portions and single tokens, over windows that the long portions cross."""
    cfg, w, g = build(name, 7)
    toks = {k: torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for k, n in (("a", 400), ("b", 40), ("c", 330))}
    want = {k: mo.forward(cfg, w, t)[0] for k, t in toks.items()}
    eng = make_engine(tmp_path, cfg, w, dtype, max_tokens=1024)
    steps = [[("a", 200), ("b", 3)], [("a", 130), ("b", 1), ("c", 129)], [("c", 200), ("a", 69), ("b", 36)], [("a", 1), ("c", 1)]]
    at, got = {k: 0 for k in toks}, {k: [] for k in toks}
    for step in steps:
        entries = []
        for k, n in step:
            entries.append((k, toks[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
        out, r = eng.step_forced(entries), 0
        for k, n in step:
            got[k].append(out.logits[r:r + n].clone())
            r += n
    for k in toks:
        assert matches(torch.cat(got[k]), want[k], dtype), k
    assert _ops().prefill_timeouts() == 0


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["base", "heads_of_64", "other_order"])
def test_mixed_batches_with_reused_pages_and_slots_equal_each_request_alone(tmp_path, dtype, name):
    """Six requests through an engine with three state slots and a small page pool: portions beside single tokens, requests that end
    and hand their pages and slot to the next one."""
    cfg, w, g = build(name, 4)
    lens = [37, 5, 61, 18, 2, 44]
    reqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lens]
    want = [mo.forward(cfg, w, t)[0] for t in reqs]
    eng = make_engine(tmp_path, cfg, w, dtype, max_tokens=160, block_size=8, live=3)
    plan = [[(0, 20), (1, 2)], [(0, 1), (1, 3), (2, 16)], [(0, 16), (2, 1)], [(2, 30), (3, 2)], [(2, 14), (3, 1), (4, 2)], [(3, 15), (5, 40)],
            [(5, 1)], [(5, 3)]]
    done, got = [0] * 6, [[] for _ in range(6)]
    for step in plan:
        entries, end = [], []
        for r, n in step:
            entries.append((f"r{r}", reqs[r][done[r]:done[r] + n], list(range(n))))
            done[r] += n
            if done[r] == lens[r]:
                end.append(f"r{r}")
        out, at = eng.step_forced(entries, end), 0
        for r, n in step:
            got[r].append(out.logits[at:at + n].clone())
            at += n
    for r in range(6):
        assert matches(torch.cat(got[r]), want[r], dtype, 1e-5, 6e-2), r
    assert done == lens and eng.cache.live == 0 and eng.cache.state_slots.num_free == 3


def test_batch_members_do_not_change_each_other(tmp_path):
    """Bit for bit: a portion alone and beside another request; a decoded token alone and beside another request's decoded token."""
    cfg, w, g = build("other_order", 5)
    a, b = (torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (33, 50))
    for dtype in BOTH:
        eng = make_engine(tmp_path, cfg, w, dtype)
        alone = [eng.step_forced([("a", a[:32], [31])]).logits.clone(), eng.step_forced([("a", a[32:], [0])], ["a"]).logits.clone()]
        both = [eng.step_forced([("b", b[:49], [48]), ("a", a[:32], [31])]).logits.clone(), eng.step_forced([("b", b[49:], [0]), ("a", a[32:], [0])], ["a", "b"]).logits.clone()]
        assert torch.equal(both[0][1], alone[0][0]) and nerr(both[1][1], alone[1][0]) < (1e-6 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
@pytest.mark.parametrize("window", [1, 2, 16, 17, 130])
def test_a_token_leaves_the_window_exactly_when_it_should(tmp_path, kind, window):
    """One layer: changing token p - window + 1 changes the logits at p, changing token p - window does not — bit for bit — in a whole
    prompt, in portions and decoded, for a p at a page's edge and one inside a page."""
    sizes = dict(mask=dict(size=window))
    cfg = mo.random_config(kinds=(kind,), mlps=("dense",), attention=sizes, latent=sizes)
    g = torch.Generator().manual_seed(31 + window)
    w = mo.random_weights(cfg, g)
    n = window + 37
    toks = torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
    eng = make_engine(tmp_path, cfg, w, torch.float32, max_tokens=512)

    def run(t, cuts):
        out, at = [], 0
        for c in cuts:
            out.append(eng.step_forced([("s", t[at:at + c], list(range(c)))], ["s"] if at + c == n else []).logits.clone())
            at += c
        return torch.cat(out)

    for cuts in ([n], [n - 35, 2, 33], [n - 9] + [1] * 9):
        base = run(toks, cuts)
        assert nerr(base, mo.forward(cfg, w, toks)[0]) < 1e-5
        for p in (n - 1, n - 6):
            inside, outside = p - window + 1, p - window
            for j, changes in ((inside, True), (outside, False)):
                t = list(toks)
                t[j] = (t[j] + 1) % cfg["vocab"]
                assert torch.equal(run(t, cuts)[p], base[p]) == (not changes), (cuts, p, j)


def test_the_first_token_is_felt_far_away_through_the_recurrence(tmp_path):
    """Slow decays (lam far below zero): changing token 0 changes the logits 300 tokens later exactly as the plain model says, whether
    the tokens came as one prompt, in portions or decoded."""
    cfg = mo.random_config(kinds=("rglru",), mlps=("dense",))
    g = torch.Generator().manual_seed(11)
    w = mo.random_weights(cfg, g)
    w["l0.mix.lam"] = bf(torch.full_like(w["l0.mix.lam"], -7.0))
    t1 = torch.randint(0, cfg["vocab"], (301,), generator=g).tolist()
    eng = make_engine(tmp_path, cfg, w, torch.float32, max_tokens=512)
    last = {}
    for name, t in (("one", t1), ("two", [(t1[0] + 1) % cfg["vocab"]] + t1[1:])):
        want = mo.forward(cfg, w, t)[0][300]
        last[name] = eng.step_forced([("a", t, [300])], ["a"]).logits[0].clone()
        assert nerr(last[name], want) < 1e-5
        for lo, hi in ((0, 2), (2, 160), (160, 299)):
            eng.step_forced([("b", t[lo:hi], [])])
        eng.step_forced([("b", t[299:300], [])])
        assert nerr(eng.step_forced([("b", t[300:], [0])], ["b"]).logits[0], want) < 1e-5
    assert nerr(last["one"], last["two"]) > 1e-4


def test_greedy_generation_through_the_scheduler(tmp_path):
    cfg, w, g = build("other_order", 6)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (19, 3, 41, 1)]
    eng = make_engine(tmp_path, cfg, w, torch.float32, max_tokens=256, block_size=8, live=2, budget=16)
    got = eng.generate(prompts, max_new_tokens=6)
    assert eng.cache.live == 0 and eng.cache.blocks.num_free == eng.cache.blocks.capacity
    for p, out in zip(prompts, got):
        assert len(out) == 6
        t = list(p)
        for tok in out:
            lg = mo.forward(cfg, w, t)[0][-1]
            top = torch.topk(lg, 2).values
            if float(top[0] - top[1]) < 1e-3:
                break
            assert int(lg.argmax()) == tok
            t.append(tok)


def test_command_line_and_trace_replay(tmp_path, capsys, monkeypatch):
    import io
    from atoma_infer_b200 import checkpoint
    from atoma_infer_b200.__main__ import main
    cfg, w, g = build("base", 8)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    checkpoint.write_safetensors(tmp_path / "model.safetensors", {k: v.to(BF) for k, v in w.items()})
    assert main(["generate", "--model", str(tmp_path), "--prompt-ids", "3,4,5,6", "--max-new-tokens", "2", "--dtype", "float32",
                 "--max-tokens", "128", "--max-live", "2"]) == 0
    line = [json.loads(x) for x in capsys.readouterr().out.strip().splitlines() if x.startswith("{")][0]
    lg = mo.forward(cfg, w, [3, 4, 5, 6])[0][-1]
    if float(torch.topk(lg, 2).values[0] - torch.topk(lg, 2).values[1]) > 1e-3:
        assert line["generated"][0] == int(lg.argmax())
    toks = [5, 9, 2, 30, 11, 7]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:4], "want": [1, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[4:5], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[5:], "want": [0]}, {"id": "b", "tokens": toks[:2], "want": [1]}], "end": ["a", "b"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    out = tmp_path / "out"
    assert main(["trace", "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "128"]) == 0
    assert [x for x in capsys.readouterr().out.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want, _ = mo.forward(cfg, w, toks)
    assert not (out / "1.f32").exists()
    a = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    b = np.fromfile(out / "2.f32", dtype="<f4").reshape(2, -1)
    assert nerr(a, want[[1, 3]]) < 1e-5 and nerr(b, torch.stack([want[5], want[1]])) < 1e-5
