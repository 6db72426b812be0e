"""Lusalorn on the GPU against the plain implementation of tests/lusalorn_oracle.py (float64): every mechanism alone, then the model
through the engine — whole prompts, token-by-token decoding, portions down to two tokens, long portions beside short ones, mixed
batches with reused pages and state slots, keys just inside and just outside every window and far away, the first tokens of a sequence,
long decoding, other sizes and layer orders, greedy generation through the scheduler and the command line."""
import json
import math

import numpy as np
import pytest
import torch

import lusalorn_oracle as lo

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
# embedding and residual stream
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("W,buckets,mul_prev,mul_cur", [(32, 101, 7, 13), (33, 5, 1, 1), (64, 1, 9, 4), (40, 1000, 999983, 1000003)])
def test_pair_embedding_on_a_mixed_batch(dtype, W, buckets, mul_prev, mul_cur):
    """Portions that start a sequence, that go on from a token of an earlier step, and single tokens."""
    g = torch.Generator().manual_seed(W)
    vocab = 50
    table, pairs = rnd(g, vocab, W), rnd(g, buckets + 1, W)
    seqs = [torch.randint(0, vocab, (n,), generator=g).tolist() for n in (9, 4, 6, 1)]
    starts = [0, 3, 2, 0]
    P = {"embed": table.double(), "bigram": pairs.double()}
    want = torch.cat([lo.embedding(s, P, dict(buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur))[a:] for s, a in zip(seqs, starts)])
    toks = i32([t for s, a in zip(seqs, starts) for t in s[a:]])
    tseq, qs = batch_layout([len(s) - a for s, a in zip(seqs, starts)])
    prev = i32([s[a - 1] if a else -1 for s, a in zip(seqs, starts)])
    x, h = _ops().embed_pairs(toks, tseq, qs, prev, table.to(dtype).to(DEV), pairs.to(dtype).to(DEV), buckets, mul_prev, mul_cur)
    assert nerr(x, want) < 1e-7 and nerr(h, want) < tol(dtype, 1e-7, 4e-3)
    plain, none = _ops().embed_pairs(toks, tseq, qs, None, table.to(dtype).to(DEV), None, 0, 0, 0, want_h=False)
    assert none is None and torch.equal(plain.cpu(), table[toks.long().cpu()])


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("W,m,scale,bias", [(40, 0.7, 1.0, False), (33, 1.0, 0.6, True), (260, -0.3, 2.5, True), (128, 1.4, -1.0, False)])
def test_normed_branch_joins_the_stream(dtype, W, m, scale, bias):
    g = torch.Generator().manual_seed(W)
    T, eps = 7, 1e-3
    x, y, w, b = rnd(g, T, W), rnd(g, T, W, scale=0.1), rnd(g, W, scale=0.3), rnd(g, W, scale=0.1)
    want = lo.branch_norm(x.double(), scale * y.double() + (b.double() if bias else 0.0), m, w.double(), eps)
    xd = x.to(DEV).clone()
    h, trace = _ops().postnorm_residual(xd, w.to(DEV), 1.0, eps, dtype, y=y.to(dtype).to(DEV), want_trace=True, offset=1.0, branch_scale=m,
                                        y_bias=b.to(DEV) if bias else None, y_scale=scale)
    assert nerr(xd, want) < 1e-6 and torch.equal(xd, trace) and nerr(h, want) < tol(dtype, 1e-6, 4e-3)


# ------------------------------------------------------------------------------------------------
# rotation, norms, cache write
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,Gv,D,V,dims,scaling,bias", [(4, 2, 1, 16, 24, 8, None, True), (6, 2, 2, 24, 16, 24, dict(factor=6.0, original=128, fast=8.0, slow=1.0), False),
                                                        (2, 2, 1, 10, 12, 2, None, True), (3, 3, 3, 64, 32, 48, dict(factor=3.0, original=900, fast=24.0, slow=1.0), False)])
def test_norms_rotation_and_cache_write(dtype, H, G, Gv, D, V, dims, scaling, bias):
    """Weighted head norms before the rotation of the first dims entries in pairs (i, i + dims / 2), positions up to 200 000, fewer value
    heads than key heads, and the queries alone (no cache write)."""
    ops = _ops()
    g = torch.Generator().manual_seed(H * 100 + D)
    T, eps = 6, 1e-4
    q_off, k_off = 8, 8 + H * D + 5
    v_off = k_off + G * D + 3
    P = v_off + Gv * V + 2
    proj, b, qw, kw = rnd(g, T, P), rnd(g, P), rnd(g, D, shift=1.2, scale=0.3), rnd(g, D, shift=0.9, scale=0.3)
    pos = torch.tensor([0, 1, 5, 700, 65537, 200000])
    rot = dict(dims=dims, base=700.0, scaling=scaling)
    f, amp = lo.rotary_frequencies(rot)
    full = (proj + (b if bias else 0.0)).double()

    def head(off, n, w):
        x = lo.unit_rms(full[:, off:off + n * D].reshape(T, n, D), eps) * w.double()
        return lo.positioned(x, rot, pos)

    slots = torch.tensor([3, 0, 11, 5, -1, 7], device=DEV)
    kc, vc = torch.full((12, G, D), 9.0, dtype=dtype, device=DEV), torch.full((12, Gv, V), 9.0, dtype=dtype, device=DEV)
    args = dict(bias=b.to(DEV) if bias else None, qk_freq_lo=(f - f.float().double()).float().to(DEV), amplitude=amp, v_heads=Gv)
    q = ops.qkv_headnorm_rope_cache(proj.to(dtype).to(DEV), q_off, k_off, v_off, qw.to(DEV), kw.to(DEV), f.float().to(DEV), None, False, pos.to(DEV), slots,
                                    kc, vc, H, G, D, V, eps, **args)
    t = tol(dtype, 2e-6, 6e-3)
    assert nerr(q.reshape(T, H, D), head(q_off, H, qw)) < t
    k, v = head(k_off, G, kw), full[:, v_off:v_off + Gv * V].reshape(T, Gv, V)
    used = [i for i in range(T) if int(slots[i]) >= 0]
    at = slots[used]
    assert nerr(kc[at], k[used]) < t and nerr(vc[at], v[used]) < t
    untouched = [r for r in range(12) if r not in at.tolist()]
    assert bool((kc[untouched] == 9.0).all()) and bool((vc[untouched] == 9.0).all())
    alone = ops.qkv_headnorm_rope_cache(proj.to(dtype).to(DEV), q_off, -1, -1, qw.to(DEV), None, f.float().to(DEV), None, False, pos.to(DEV), None, None, None,
                                        H, G, D, V, eps, **args)
    assert torch.equal(alone, q)


# ------------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------------
def plain_maps(q, k, v, share, scale, window, start):
    """[n, H, V] of the queries start .. start + n - 1 (q) against keys 0 .. start + n - 1."""
    H, G = q.shape[1], k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, 1)) * scale
    d = (start + torch.arange(q.shape[0]))[:, None] - torch.arange(k.shape[0])[None, :]
    s = s.masked_fill((d < 0) | ((d >= window) if window else (d < 0)), -math.inf)
    return torch.einsum("hij,jhv->ihv", torch.softmax(s, -1), v.repeat_interleave(share, 1).repeat_interleave(H // G, 1))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,share,D,V,window,long_", [(4, 2, 2, 16, 32, 9, 0), (6, 2, 2, 48, 80, 41, 0), (8, 2, 2, 64, 128, 33, 128), (4, 4, 2, 64, 64, 0, 128),
                                                       (4, 4, 2, 48, 128, 130, 128), (8, 4, 2, 128, 128, 150, 128), (2, 2, 1, 64, 128, 0, 128), (3, 3, 3, 10, 14, 7, 0),
                                                       (4, 2, 2, 96, 64, 70, 128), (20, 1, 1, 32, 48, 0, 0), (6, 6, 3, 80, 112, 100, 0)])
def test_softmax_attention_with_shared_value_heads(dtype, H, G, share, D, V, window, long_):
    """Neighbouring key heads read one value head, keys and values of different sizes, an output row wider than the heads; a mixed batch of
    single tokens, short and (long_) long portions, sequences on shuffled pages."""
    ops = _ops()
    g = torch.Generator().manual_seed(H * 1000 + D)
    seqs, bs = [(0, 150), (37, 1), (20, 135), (16, 2), (300, 1), (3, 70)], 16
    lens = [c + n for c, n in seqs]
    bt, rows, n_rows = paged(lens, bs, g)
    kc, vc = torch.full((n_rows, G, D), 30.0, dtype=dtype, device=DEV), torch.full((n_rows, G // share, V), 30.0, dtype=dtype, device=DEV)
    ks, vs = [rnd(g, n, G, D) for n in lens], [rnd(g, n, G // share, V) for n in lens]
    for b in range(len(seqs)):
        idx = torch.tensor(rows[b], device=DEV)
        kc[idx], vc[idx] = ks[b].to(dtype).to(DEV), vs[b].to(dtype).to(DEV)
    T, scale = sum(n for _, n in seqs), 1.6 / math.sqrt(D)
    q = rnd(g, T, H, D)
    tseq, qs = batch_layout([n for _, n in seqs])
    pos = torch.tensor([c + i for c, n in seqs for i in range(n)], device=DEV)
    wide = torch.full((T, H * V + 16), 5.0, dtype=dtype, device=DEV)
    ops.softmax_attention_paged(q.reshape(T, -1).to(dtype).to(DEV), kc, vc, pos, tseq, bt.to(DEV), H, G, D, V, bs, scale, window=window, query_start=qs,
                                long_min_q=long_, out=wide[:, :H * V], v_share=share)
    assert bool((wide[:, H * V:] == 5.0).all())
    at = 0
    for b, (c, n) in enumerate(seqs):
        want = plain_maps(q[at:at + n].double(), ks[b].double(), vs[b].double(), share, scale, window, c)
        assert nerr(wide[at:at + n, :H * V].reshape(n, H, V), want) < tol(dtype, 1e-5, 1.5e-2), b
        at += n
    assert ops.prefill_timeouts() == 0


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,V,lam,diff", [(4, 2, 24, 0.4, 0.3), (6, 1, 7, -0.7, 0.1), (3, 3, 128, 1.2, 0.8), (1, 1, 1, 0.0, 0.5), (8, 2, 300, 0.9, -0.2)])
def test_two_maps_into_one(dtype, H, G, V, lam, diff):
    g = torch.Generator().manual_seed(V)
    T, eps, rep = 5, 1e-4, H // G
    maps = rnd(g, T, 2, H, V)
    want = lo.combine_maps(maps[:, 0].double(), maps[:, 1].double(), lam, diff, eps)
    grouped = maps.reshape(T, 2, G, rep, V).permute(0, 2, 1, 3, 4).reshape(T, 2 * H * V).contiguous()
    got = _ops().differential_combine(grouped.to(dtype).to(DEV), H, G, V, lam, 1.0 - diff, eps)
    assert nerr(got.reshape(T, H, V), want) < tol(dtype, 2e-6, 4e-3)


@pytest.mark.parametrize("mode", ["decoded", "short", "long"])
@pytest.mark.parametrize("far", [1, 15, 16, 17, 63, 64, 127, 128, 200, 511])
def test_one_loud_key_at_the_edge_of_the_window(mode, far):
    """One key's score stands far above the rest.  A query `far` tokens later reads (only) its value through a window of far + 1 tokens and
    nothing of it through a window of far tokens — keys of 64 under values of 128 that two key heads share."""
    ops = _ops()
    g = torch.Generator().manual_seed(far)
    D, V, bs, before = 64, 128, 16, 40
    n = before + far + 1
    count = {"decoded": 1, "short": 2, "long": max(150, far + 2)}[mode]
    if count > n:
        before, n = before + count - n, count
    loud = before
    bt, rows, n_rows = paged([n], bs, g)
    idx = torch.tensor(rows[0], device=DEV)
    k, v = rnd(g, n, 2, D, scale=0.01), rnd(g, n, 1, V)
    k[loud, 1] = 0
    k[loud, 1, 5] = 16.0
    q = torch.zeros(count, 2, D)
    q[-1, 1, 5] = 16.0
    kc, vc = torch.zeros((n_rows, 2, D), dtype=BF, device=DEV), torch.zeros((n_rows, 1, V), dtype=BF, device=DEV)
    kc[idx], vc[idx] = k.to(BF).to(DEV), v.to(BF).to(DEV)
    for window, seen in ((far + 1, True), (far, False), (0, True)):
        out = ops.softmax_attention_paged(q.reshape(count, -1).to(BF).to(DEV), kc, vc, torch.arange(n - count, n, device=DEV), i32([0] * count), bt.to(DEV), 2, 2,
                                          D, V, bs, 1.0, window=window, query_start=i32([0, count]), long_min_q=128, v_share=2)
        got = out.reshape(count, 2, V)[-1, 1].double().cpu()
        want = plain_maps(q[-1:].double(), k.double(), v.double(), 2, 1.0, window, n - 1)[0, 1]
        assert float((got - want).abs().max()) < 3e-2
        assert (float((got - v[loud, 0].double()).abs().max()) < 3e-2) == seen, window


# ------------------------------------------------------------------------------------------------
# state-space recurrence
# ------------------------------------------------------------------------------------------------
def ssm_case(g, H, G, N, V, n):
    return dict(x=rnd(g, n, H * V), B=rnd(g, n, G * N, scale=0.5), C=rnd(g, n, G * N), dt=rnd(g, n, H, shift=-1.0))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,N,V,flags", [(4, 2, 16, 8, 0), (6, 3, 20, 12, 0), (2, 1, 128, 64, 0), (2, 1, 128, 64, 16), (3, 3, 64, 40, 16), (8, 4, 40, 24, 0), (1, 1, 300, 9, 0),
                                           (5, 1, 7, 33, 0), (2, 2, 200, 16, 16), (4, 4, 256, 64, 0)])
def test_state_space_scan_over_portions_and_reused_slots(dtype, H, G, N, V, flags):
    """Portions down to one token on slots that hold garbage of earlier requests; step sizes from tiny to above 20 before the softplus;
    groups of heads; both splits of the rows over lanes; long portions beside single tokens."""
    ops = _ops()
    ops.debug_flags(flags)
    g = torch.Generator().manual_seed(H * 100 + N)
    lens = [45, 290, 6]
    cases = [ssm_case(g, H, G, N, V, n) for n in lens]
    for c in cases:
        c["dt"][2] = 21.5
        c["dt"][3] = -12.0
    a_log, dtb, skip = rnd(g, H, shift=-0.5), rnd(g, H, scale=0.5), rnd(g, H)
    want = [lo.state_space(c["x"].double().reshape(-1, H, V), c["B"].double().reshape(-1, G, N), c["C"].double().reshape(-1, G, N),
                           lo.softplus(c["dt"].double() + dtb.double()), a_log.double(), skip.double()).reshape(-1, H * V) for c in cases]
    state = torch.full((4, H * N * V + 3), 1e3, device=DEV)
    slots, done, got = [2, 0, 3], [0, 0, 0], [[], [], []]
    for step in ([(0, 20), (1, 2)], [(0, 1), (1, 160), (2, 2)], [(2, 1), (0, 24)], [(1, 128), (2, 3)]):
        ctx = i32([done[b] for b, _ in step])
        part = {k: torch.cat([cases[b][k][done[b]:done[b] + n] for b, n in step]).to(dtype).to(DEV) for k in ("x", "B", "C", "dt")}
        _, qs = batch_layout([n for _, n in step])
        out = ops.ssm_scan(part["x"], part["B"], part["C"], part["dt"], a_log.to(DEV), dtb.to(DEV), skip.to(DEV), state, i32([slots[b] for b, _ in step]), qs, ctx,
                           H, G, N, V)
        at = 0
        for b, n in step:
            got[b].append(out[at:at + n])
            at += n
            done[b] += n
    assert done == lens
    for b in range(3):
        assert nerr(torch.cat(got[b]), want[b]) < 2e-5, b      # inputs are exact in both formats, everything after them is float32
    assert bool((state[1] == 1e3).all()) and bool((state[:, H * N * V:] == 1e3).all())


@pytest.mark.parametrize("dtype", BOTH)
def test_state_space_scan_keeps_a_write_for_hundreds_of_tokens(dtype):
    """Decay close to one: a single loud write is read 600 tokens later with the product of all decays; a head with strong decay
    has forgotten it."""
    ops = _ops()
    H, G, N, V, n = 2, 1, 32, 16, 601
    x, B, C = torch.zeros(n, H * V), torch.zeros(n, G * N), torch.zeros(n, G * N)
    x[0], B[0, 3], C[-1, 3] = 8.0, 4.0, 1.0
    g = torch.Generator().manual_seed(3)
    dt, a_log = rnd(g, n, H, scale=0.7, shift=-5.0), torch.tensor([-3.0, 6.0])     # (constant decays would add their rounding up)
    want = lo.state_space(x.double().reshape(n, H, V), B.double().reshape(n, G, N), C.double().reshape(n, G, N), lo.softplus(dt.double()), a_log.double(),
                          torch.zeros(H, dtype=F64))[-1]
    assert float(want[0, 0]) > 0.05 and float(want[1, 0]) < 1e-12
    for cuts in ([601], [300, 301], [2, 598, 1], [1, 127, 128, 344, 1]):
        state, at = torch.full((1, H * N * V), 7.0, device=DEV), 0
        for c in cuts:
            sl = slice(at, at + c)
            dv = lambda t: t[sl].to(dtype).to(DEV)
            out = ops.ssm_scan(dv(x), dv(B), dv(C), dv(dt), a_log.to(DEV), torch.zeros(H, device=DEV), None, state, i32([0]), i32([0, c]), i32([at]), H, G, N, V)
            at += c
        got = out[-1].reshape(H, V)
        assert nerr(got[0], want[0]) < 3e-5 and float(got[1].abs().max()) < 1e-10, cuts


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("n,parts,before,after", [(72, 2, 0, 0), (30, 3, 2, 6), (256, 1, 0, 8), (1024, 4, 8, 0), (36, 12, 4, 4), (35, 5, 1, 0), (2048, 8, 0, 0), (22, 11, 0, 2)])
def test_gate_before_the_grouped_norm(dtype, n, parts, before, after):
    g = torch.Generator().manual_seed(n + parts)
    T, eps = 5, 1e-3
    o, z, w = torch.randn(T, n, generator=g) * 0.3, rnd(g, T, n + 8), rnd(g, n, shift=1.0, scale=0.3)
    want = lo.gate_then_norm(o.double(), z[:, :n].double(), w.double(), parts, eps)
    wide = torch.full((T, 8 + before + n + after + 8), 3.0, dtype=dtype, device=DEV)
    view = wide[:, 8 + before:8 + before + n]
    _ops().gate_groupnorm(o.to(DEV), z.to(dtype).to(DEV), w.to(DEV), parts, eps, out=view, zero_before=before, zero_after=after)
    assert nerr(view, want) < tol(dtype, 2e-6, 4e-3)
    assert bool((wide[:, :8] == 3.0).all()) and bool((wide[:, 8 + before + n + after:] == 3.0).all())
    assert bool((wide[:, 8:8 + before] == 0).all()) and bool((wide[:, 8 + before + n:8 + before + n + after] == 0).all())


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
    "other_order": dict(kinds=("attention", "attention", "shared", "parallel", "shared", "parallel"), mlps=(True, False, True, False, False, True), mult=1.3, eps=1e-3,
                        shared=dict(heads=6, scale=0.2, diff=0.6, mask=dict(size=9)), scales=(-0.8, 0.4)),
    "no_state": dict(kinds=("attention", "shared"), attention=dict(mask=dict(size=1)), shared=dict(mask=dict(size=300))),
    "only_parallel": dict(kinds=("parallel", "parallel"), mlps=False, bigram=None, scales=(1.0, 1.0), mult=1.0),
    "odd_sizes": dict(width=50, vocab=37, ff=22, mult=0.4, kinds=("parallel", "attention", "parallel", "shared"), bigram=(13, 1009, 3),
                      attention=dict(heads=6, kv_heads=3, dim=12, vdim=10, scale=0.4, diff=0.15, mask=dict(size=5), rot=dict(base=90.0, dims=12)),
                      left=dict(heads=3, kv_heads=1, dim=10, vdim=14, scale=0.5, rot=dict(base=777.0, dims=6, scaling=dict(factor=2.0, original=50, fast=3.0, slow=1.0))),
                      right=dict(heads=6, vdim=5, groups=2, state=9, norm_groups=5, conv=3)),
    "one_of_each": dict(kinds=("parallel", "attention"), attention=dict(heads=1, kv_heads=1, dim=16, vdim=16, mask=dict(size=2), rot=dict(base=50.0, dims=2)),
                        left=dict(heads=1, kv_heads=1, dim=16, vdim=16), right=dict(heads=1, vdim=24, groups=1, state=8, norm_groups=1, conv=1), bigram=(1, 1, 1)),
    "heads_of_64": dict(width=64, kinds=("parallel", "attention", "shared", "parallel"),
                        attention=dict(heads=4, kv_heads=2, dim=64, vdim=128, scale=0.125, mask=dict(size=50), rot=dict(base=1e4, dims=32)),
                        left=dict(heads=4, kv_heads=1, dim=64, vdim=64, scale=0.125, rot=dict(base=1e5, dims=64, scaling=dict(factor=4.0, original=64, fast=16.0, slow=1.0))),
                        right=dict(heads=4, vdim=64, groups=2, state=64, norm_groups=4, conv=4)),
    "heads_of_128": dict(width=64, kinds=("attention", "parallel"),
                         attention=dict(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.09, mask=dict(size=300), rot=dict(base=1e4, dims=64)),
                         left=dict(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.09), right=dict(heads=2, vdim=64, groups=1, state=128, norm_groups=1, conv=4)),
    "left_off": dict(kinds=("parallel",), scales=(0.0, 1.5)),
    "right_off": dict(kinds=("parallel",), scales=(1.5, 0.0)),
}


def build(name, seed=0):
    g = torch.Generator().manual_seed(700 + seed)
    cfg = lo.random_config(**VARIANTS[name])
    return cfg, lo.random_weights(cfg, g), g


def matches(got, want, dtype, f32=1e-5, bf16=4e-2):
    return nerr(got, want) < (f32 if dtype == torch.float32 else bf16)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", list(VARIANTS))
def test_whole_prompt_matches_the_plain_model(tmp_path, dtype, name):
    cfg, w, g = build(name)
    toks = torch.randint(0, cfg["vocab"], (83,), generator=g).tolist()
    want, layers = lo.forward(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, dtype)
    out = eng.step_forced([("a", toks, list(range(len(toks))))], want_residual_trace=True)
    assert out.residual_trace.shape[0] == len(layers)
    for i in range(len(layers)):
        assert matches(out.residual_trace[i], layers[i], dtype, 5e-6, 3e-2), (i, nerr(out.residual_trace[i], layers[i]))
    assert matches(out.logits, want, dtype), nerr(out.logits, want)


@pytest.mark.parametrize("name", list(VARIANTS))
def test_decoding_token_by_token_equals_the_whole_prompt(tmp_path, name):
    """90 single-token steps on pages of four tokens: every page border, the first tokens of the sequence (where the filter still looks
    before its start and the pair table has a row of its own), windows that fill up and then slide."""
    cfg, w, g = build(name, 1)
    toks = torch.randint(0, cfg["vocab"], (90,), generator=g).tolist()
    want, _ = lo.forward(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, torch.float32, max_tokens=128, block_size=4)
    got = [eng.step_forced([("a", [t], [0])]).logits.clone() for t in toks]
    assert nerr(torch.cat(got), want) < 1e-5


def test_long_decoding(tmp_path):
    """A short prompt and 400 decoded tokens: the state is carried for hundreds of steps, the windows slide over many pages."""
    cfg, w, g = build("base", 2)
    toks = torch.randint(0, cfg["vocab"], (420,), generator=g).tolist()
    want, _ = lo.forward(cfg, w, toks)
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
    want, _ = lo.forward(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, dtype, max_tokens=256, block_size=8)
    got, at = [], 0
    for n in sizes:
        got.append(eng.step_forced([("a", toks[at:at + n], list(range(n)))]).logits.clone())
        at += n
    assert matches(torch.cat(got), want, dtype)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["heads_of_64", "heads_of_128", "base"])
def test_long_portions_beside_short_ones_and_decoded_tokens(tmp_path, dtype, name):
    """Portions of 128 tokens and more (bfloat16 heads of 64 / 128: the tensor-memory attention kernel) in one step with short portions
    and single tokens, over windows that the long portions cross."""
    cfg, w, g = build(name, 7)
    toks = {k: torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for k, n in (("a", 400), ("b", 40), ("c", 330))}
    want = {k: lo.forward(cfg, w, t)[0] for k, t in toks.items()}
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
    """Six requests through an engine with three state slots and a small page pool: portions beside single tokens, requests that pause, that
    end and hand their pages and slot to the next one."""
    cfg, w, g = build(name, 4)
    lens = [37, 5, 61, 18, 2, 44]
    reqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lens]
    want = [lo.forward(cfg, w, t)[0] for t in reqs]
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
        assert matches(torch.cat(got[r]), want[r], dtype, 1e-5, 5e-2), r
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


@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("window", [1, 2, 16, 17, 130])
def test_a_token_leaves_the_window_exactly_when_it_should(tmp_path, shared, window):
    """Changing token p - window + 1 changes the logits at p, changing token p - window does not — bit for bit — in a whole prompt, in
    portions and decoded, for a p at a page's edge and one inside a page.  `shared`: the window is that of a layer on another layer's keys
    and values, whose own window is one token.  (No pair table: it would carry a token one place further.)"""
    if shared:
        cfg = lo.random_config(kinds=("attention", "shared"), attention=dict(mask=dict(size=1)), shared=dict(mask=dict(size=window)), bigram=None)
    else:
        cfg = lo.random_config(kinds=("attention",), attention=dict(mask=dict(size=window)), bigram=None)
    g = torch.Generator().manual_seed(31 + window)
    w = lo.random_weights(cfg, g)
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
        assert nerr(base, lo.forward(cfg, w, toks)[0]) < 1e-5
        for p in (n - 1, n - 6):
            inside, outside = p - window + 1, p - window
            for j, changes in ((inside, True), (outside, False)):
                t = list(toks)
                t[j] = (t[j] + 1) % cfg["vocab"]
                assert torch.equal(run(t, cuts)[p], base[p]) == (not changes), (cuts, p, j)


def loudest_last_token(cfg, w, toks):
    """The last token whose query (some head's) gives the first key the largest softmax weight in a one-layer model."""
    P, m, pre, eps, n = {k: v.double() for k, v in w.items()}, cfg["layers"][0]["mixer"]["left"], "l0.mix.left.", cfg["norm"]["eps"], len(toks)

    def heads(x, name, count, positions):
        return lo.positioned(lo.unit_rms((x @ P[pre + name].T).reshape(len(x), count, m["dim"]), eps) * P[pre + name + ".norm"], m["rot"], positions)

    def weight(tok):
        x = lo.embedding(toks[:-1] + [tok], P, cfg["embedding"]["bigram"])
        k, q = heads(x, "k", m["kv_heads"], range(n)), heads(x[-1:], "q", m["heads"], [n - 1])[0]
        per = m["heads"] // m["kv_heads"]
        return max(float(torch.softmax(k[:, h // per] @ q[h] * m["scale"], 0)[0]) for h in range(m["heads"]))

    return max(range(cfg["vocab"]), key=weight)


@pytest.mark.parametrize("side", ["attention", "recurrence"])
def test_the_first_token_is_felt_far_away(tmp_path, side):
    """Changing token 0 changes the logits 300 tokens later exactly as the plain model says — through a loud key of the full attention, or
    through slow decays of the recurrence — whether the tokens came as one prompt, in portions or decoded."""
    cfg = lo.random_config(kinds=("parallel",), mlps=True, scales=(1.0, 0.0) if side == "attention" else (0.0, 1.0))
    g = torch.Generator().manual_seed(11)
    w = lo.random_weights(cfg, g)
    if side == "recurrence":
        w["l0.mix.right.A_log"] = torch.full_like(w["l0.mix.right.A_log"], -7.0)
    else:
        w["l0.mix.left.q.norm"], w["l0.mix.left.k.norm"] = bf(w["l0.mix.left.q.norm"] * 2), bf(w["l0.mix.left.k.norm"] * 2)
    t1 = torch.randint(0, cfg["vocab"], (301,), generator=g).tolist()
    if side == "attention":
        t1 = t1[:300] + [loudest_last_token(cfg, w, t1)]
    eng = make_engine(tmp_path, cfg, w, torch.float32, max_tokens=512)
    last = {}
    for name, t in (("one", t1), ("two", [(t1[0] + 1) % cfg["vocab"]] + t1[1:])):
        want = lo.forward(cfg, w, t)[0][300]
        last[name] = eng.step_forced([("a", t, [300])], ["a"]).logits[0].clone()
        assert nerr(last[name], want) < 1e-5
        for a, b in ((0, 2), (2, 160), (160, 299)):
            eng.step_forced([("b", t[a:b], [])])
        eng.step_forced([("b", t[299:300], [])])
        assert nerr(eng.step_forced([("b", t[300:], [0])], ["b"]).logits[0], want) < 1e-5
    assert nerr(last["one"], last["two"]) > 5e-5


def test_the_token_before_a_portion_is_carried(tmp_path):
    """The pair table alone (a window of one token, no state): the logits of a portion's first token depend on the token before it, the same
    whether that token was in this step or an earlier one; a sequence's first token reads the last row."""
    cfg = lo.random_config(kinds=("attention",), attention=dict(mask=dict(size=1)), bigram=(53, 17, 29))
    g = torch.Generator().manual_seed(5)
    w = lo.random_weights(cfg, g)
    toks = torch.randint(0, cfg["vocab"], (40,), generator=g).tolist()
    want = lo.forward(cfg, w, toks)[0]
    assert nerr(lo.forward(cfg, w, toks[7:8])[0], want[7:8]) > 1e-2
    for sizes in ([40], [1] * 40, [2] * 20, [7, 1, 9, 16, 2, 5]):
        eng = make_engine(tmp_path, cfg, w, torch.float32, max_tokens=128, block_size=8)
        got, at = [], 0
        for n in sizes:
            got.append(eng.step_forced([("a", toks[at:at + n], list(range(n)))]).logits.clone())
            at += n
        assert nerr(torch.cat(got), want) < 1e-5, sizes


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
            lg = lo.forward(cfg, w, t)[0][-1]
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
    lg = lo.forward(cfg, w, [3, 4, 5, 6])[0][-1]
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
    want, _ = lo.forward(cfg, w, toks)
    assert not (out / "1.f32").exists()
    a = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    b = np.fromfile(out / "2.f32", dtype="<f4").reshape(2, -1)
    assert nerr(a, want[[1, 3]]) < 1e-5 and nerr(b, torch.stack([want[5], want[1]])) < 1e-5
