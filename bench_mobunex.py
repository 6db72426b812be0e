"""bench.py --design mobunex: prefill and decode throughput of the Mobunex design (random weights) at sizes that resemble real models'
layers, beside the framework's closest existing model — Nemasun, the other design of windowed softmax attention and mixtures of experts
with a restricted choice — at equal width, head counts, head size, window, feed-forward sizes and number of layers, and the design's own
kernels against the measured peaks beside the like kernels of the models they come from (Nemasun's attention, norms and router, Patadra's
latent attention and per-head products, Lilovik's recurrence, Surinex's filter).  Not the headline (config 2 is); ONE JSON line in the
same format.

Per size: `prefill` = one 4096-token prompt in one step; `decode` = one step of 32 sequences at context 4096 (built by prefilling them),
timed with CUDA events around K executor steps after W warm-up steps, inputs shipped from pinned memory every step, sampled tokens read
back; the same step replayed from a CUDA graph is the device-only figure.  Kernel rows: achieved bytes/s or FLOP/s over the measured peaks
of MEASURED_PEAKS.json (fallback figures when absent); L2 is flushed between their iterations."""
from __future__ import annotations

import json
import math
import os
import time

import bench_nemasun
from bench_hybrid import BATCH, CTX, PROMPT, _peaks, _time
from bench_patadra import _row

SIZES = {
    "2k-wide": dict(width=2048, vocab=32000, alpha=2.0, window=1024, ff=8192, attention=dict(heads=32, kv_heads=8, dim=64),
                    latent=dict(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=512), lru=dict(width=2560, blocks=10, taps=4),
                    experts=32, top=4, expert_ff=1024, shared_ff=2048, groups=4, keep_groups=2,
                    layers=(("latent", "dense"), ("attention", "moe"), ("lru", "dense"), ("attention", "moe"))),
    "4k-wide": dict(width=4096, vocab=32000, alpha=2.0, window=4096, ff=14336, attention=dict(heads=32, kv_heads=8, dim=128),
                    latent=dict(heads=32, dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512), lru=dict(width=4096, blocks=16, taps=4),
                    experts=64, top=6, expert_ff=1408, shared_ff=2816, groups=8, keep_groups=4,
                    layers=(("latent", "dense"), ("attention", "moe"), ("lru", "dense"))),
}


def _spec(s):
    from atoma_infer_b200.hybrid import (HybridSpec, LatentAttentionSpec, LayerSpec, LinearRecurrentSpec, MlpSpec, MoeSpec, RotarySpec, SoftmaxAttentionSpec)
    a, l, d = s["attention"], s["latent"], s["lru"]
    mixers = {
        "attention": dict(mixer="softmax_attention", softmax=SoftmaxAttentionSpec(a["heads"], a["kv_heads"], a["dim"], a["dim"], 1 / math.sqrt(a["dim"]), s["window"],
                                                                                  bias=True, head_scale=True)),
        "latent": dict(mixer="latent_attention",
                       latent=LatentAttentionSpec(l["heads"], l["dim"], l["vdim"], l["q_rank"], l["kv_rank"], 1 / math.sqrt(l["dim"] + l["rot_dim"]), s["window"],
                                                  rot_dim=l["rot_dim"], rotary=RotarySpec(l["rot_dim"], 1e5, True, yarn=(8.0, 4096, 32.0, 1.0)), out_gate=True)),
        "lru": dict(mixer="lru", lru=LinearRecurrentSpec(d["width"], d["blocks"], d["taps"])),
    }
    ffs = {
        "dense": dict(mlp=MlpSpec(s["ff"], "silu")),
        "moe": dict(moe=MoeSpec(experts=s["experts"], top=s["top"], ff=s["expert_ff"], shared_ff=s["shared_ff"], alpha=1.0, up_shift=0.0, renormalize=True,
                                correction=True, groups=s["groups"], keep_groups=s["keep_groups"], group_top=2, scale_input=False)),
    }
    return HybridSpec(s["width"], s["vocab"], 1e-5, 1.0, tuple(LayerSpec(**mixers[m], **ffs[f]) for m, f in s["layers"]), norm_offset=0.0,
                      block_style="postnorm", position="none", residual_alpha=s["alpha"], depth_average=True)


def _weights(torch, spec, s, dev):
    gen = torch.Generator(device=dev).manual_seed(19)

    def r(*shape, scale=1.0, mean=0.0):
        return (mean + torch.randn(shape, generator=gen, device=dev, dtype=torch.float32) * scale).to(torch.bfloat16)

    W = spec.width
    lin = lambda o, i: r(o, i, scale=i ** -0.5)
    one = lambda: torch.ones(W, device=dev)
    out = {"embed": r(spec.vocab, W), "head": lin(spec.vocab, W), "embed_norm": one(), "final_norm": one(), "layers": []}
    for i, ls in enumerate(spec.layers):
        w = {"norm1": one(), "norm2": one(), "depth_w": torch.full((i + 2,), 0.1)}
        w["depth_w"][-1] = 1.0
        if ls.softmax is not None:
            a = ls.softmax
            nq, nk = a.heads * a.dim, a.kv_heads * a.dim
            w.update(w_q=lin(nq, W), w_k=lin(nk, W), w_v=lin(nk, W), b_q=r(nq, scale=0.1), b_k=r(nk, scale=0.1), b_v=r(nk, scale=0.1),
                     head_scale=r(a.heads, scale=0.1, mean=1.0), w_o=lin(W, nq))
        elif ls.latent is not None:
            a = ls.latent
            w.update(w_dq=lin(a.q_rank, W), dq_norm=r(a.q_rank, scale=0.1, mean=1.0), w_uq=lin(a.heads * (a.dim + a.rot_dim), a.q_rank),
                     w_dkv=lin(a.kv_rank + a.rot_dim, W), dkv_norm=r(a.kv_rank, scale=0.1, mean=1.0), w_uk=lin(a.heads * a.dim, a.kv_rank),
                     w_uv=lin(a.heads * a.vdim, a.kv_rank), w_g=lin(a.heads * a.vdim, W), w_o=lin(W, a.heads * a.vdim))
        else:
            d = ls.lru
            S, n = d.width, d.width // d.blocks
            w.update(w_y=lin(S, W), w_x=lin(S, W), b_y=r(S, scale=0.1), b_x=r(S, scale=0.1), tap_w=r(S, d.taps, scale=0.5), tap_b=r(S, scale=0.1),
                     gate_r=r(d.blocks, n, n, scale=n ** -0.5), gate_i=r(d.blocks, n, n, scale=n ** -0.5), gate_r_b=r(S), gate_i_b=r(S),
                     rate=-torch.rand(S, generator=gen, device=dev) * 0.5, w_o=lin(W, S))
        if ls.mlp is not None:
            w.update(w_gate_up=lin(2 * ls.mlp.ff, W), w_down=lin(W, ls.mlp.ff))
        if ls.moe is not None:
            e = ls.moe
            w.update(w_router=lin(e.experts, W), router_correction=r(e.experts, scale=0.01), w_expert_gate_up=r(e.experts, 2 * e.ff, W, scale=W ** -0.5),
                     w_expert_down=r(e.experts, W, e.ff, scale=e.ff ** -0.5), w_ff_in=lin(2 * e.shared_ff, W), w_down=lin(W, e.shared_ff))
        out["layers"].append(w)
    return out


def _nemasun_sizes(s):
    """A Nemasun model of equal width, heads, head size, window, feed-forward sizes and number of layers."""
    a = s["attention"]
    return dict(width=s["width"], lanes=4, heads=a["heads"], kv_heads=a["kv_heads"], dim=a["dim"], window=s["window"], keep=4, table_rows=512, ff=s["ff"],
                limit=7.0, experts=s["experts"], identity=0, top=s["top"], groups=s["groups"], keep_groups=s["keep_groups"], expert_ff=s["expert_ff"],
                shared_ff=s["shared_ff"], vocab=s["vocab"], kinds=tuple(f for _, f in s["layers"]))


def _serve(torch, spec, weights, dev, steps, warmup):
    """Prefill and decode of a model through the engine's executor."""
    import numpy as np
    from atoma_infer_b200.cache import CacheManager
    from atoma_infer_b200.engine import Engine
    from atoma_infer_b200.hybrid import HybridExecutor, relaunch_last_step
    page = 16
    nblocks, slots = BATCH * ((CTX + 64) // page + 1) + PROMPT // page + 8, BATCH + 1 if spec.has_state else 0
    ex = HybridExecutor(spec, weights, torch.bfloat16, dev, nblocks, page, slots)
    eng = Engine(ex, CacheManager(nblocks, page, slots), max_num_batched_tokens=PROMPT, max_num_seqs=BATCH + 1)
    rng = np.random.default_rng(0)
    prompt = rng.integers(0, spec.vocab, size=PROMPT).tolist()

    def prefill():
        eng.step_forced([("p", prompt, [PROMPT - 1])], end=["p"]).next_tokens.cpu()
    ms_prefill = _time(torch, prefill, min(steps, 10), warmup)
    prefill_launches = ex.launches_last_step
    for b in range(BATCH):
        eng.step_forced([(f"d{b}", rng.integers(0, spec.vocab, size=CTX).tolist(), [])])
    tok = [int(t) for t in rng.integers(0, spec.vocab, size=BATCH)]

    def decode():
        eng.step_forced([(f"d{b}", [tok[b]], [0]) for b in range(BATCH)]).next_tokens.cpu()
    ms_decode = _time(torch, decode, min(steps, 40), warmup)
    launches = ex.launches_last_step
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        relaunch_last_step(ex)
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph, stream=side):
        relaunch_last_step(ex)
    ms_graph = _time(torch, graph.replay, steps, warmup)
    del graph, eng, ex
    torch.cuda.empty_cache()
    return dict(prefill_ms=round(ms_prefill, 3), prefill_tokens_per_s=round(PROMPT / ms_prefill * 1e3, 1), prefill_launches=prefill_launches,
                decode_ms_per_step=round(ms_decode, 4), decode_tokens_per_s=round(BATCH / ms_decode * 1e3, 1), decode_graph_ms_per_step=round(ms_graph, 4),
                decode_graph_tokens_per_s=round(BATCH / ms_graph * 1e3, 1), decode_launches_per_step=launches)


def _kernel_rows(torch, s, dev, steps, warmup, hbm, tf):
    """The design's kernels beside the like kernels of the models they come from, at the same shapes."""
    from atoma_infer_b200 import hybrid_ops as ho
    bf, W, win, page = torch.bfloat16, s["width"], s["window"], 16
    rows = {}
    flush = torch.empty(160 << 20, dtype=torch.uint8, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    rn = lambda *shape: torch.randn(shape, device=dev, dtype=bf)

    def put(key, f, **kw):
        rows[key] = _row(_time(torch, f, steps, warmup, flush), hbm=hbm, tf=tf, **kw)

    a, l, d = s["attention"], s["latent"], s["lru"]
    H, G, D = a["heads"], a["kv_heads"], a["dim"]
    LH, LD, Rd, LV, Rk = l["heads"], l["dim"], l["rot_dim"], l["vdim"], l["kv_rank"]
    R = Rk + Rd
    table = torch.randn((512, H), device=dev) * 0.5
    # ---- attention: one 4096-token prompt, and a decode step of BATCH sequences at context CTX ----
    for name, T, B, ctx in (("prefill", PROMPT, 1, 0), ("decode", BATCH, BATCH, CTX)):
        n = T // B
        mb = (ctx + n + page - 1) // page
        bt = torch.randperm(B * mb, device=dev).to(torch.int32).reshape(B, mb)
        pos = (torch.arange(n, device=dev) + ctx).repeat(B)
        tseq, qs = torch.arange(B, device=dev, dtype=torch.int32).repeat_interleave(n), i32([i * n for i in range(B + 1)])
        pairs = B * sum(min(ctx + i + 1, win) for i in range(n))
        keys = B * min(ctx + n, win + n - 1)
        kc, vc, q, gate = rn(B * mb * page, G, D), rn(B * mb * page, G, D), rn(T, H * D), rn(T, H * D)
        kw = dict(window=win, max_query_len=n, query_start=qs, max_seq_len=ctx + n)
        if name == "prefill":
            kw.update(long_min_q=128, long_stats=(1, T, 0))
        mine = lambda: ho.softmax_attention_paged(q, kc, vc, pos, tseq, bt, H, G, D, D, page, D ** -0.5, **kw)
        like = lambda: ho.softmax_attention_paged(q, kc, vc, pos, tseq, bt, H, G, D, D, page, D ** -0.5, keep_first=4, dist_bias=table, gate=gate, **kw)
        for key, f in ((f"softmax_attention_{name}", mine), (f"nemasun_softmax_attention_{name}", like)):
            put(key, f, flops=4.0 * pairs * H * D, nbytes=keys * G * 2 * D * 2)
        del kc, vc, q, gate
        cache, og = rn(B * mb * page, R), rn(T, LH * LV)
        plain = cache[:, :Rk].contiguous()
        if name == "prefill":
            wk, wv, ws = rn(LH * (LD + Rd), R) * R ** -0.5, rn(LH * LV, Rk) * Rk ** -0.5, rn(LH * LD, Rk) * Rk ** -0.5
            q, qp, ctx0, sink = rn(T, LH * (LD + Rd)), rn(T, LH * LD), i32([0]), torch.zeros(LH, device=dev)
            o = torch.empty((T, LH * LV), device=dev, dtype=bf)
            f = lambda: ho.latent_attention_expanded(q, cache, wk, wv, qs, ctx0, bt, None, LH, LD, Rk, page, win, (LD + Rd) ** -0.5, 128, T, T, T, out=o, rot_dim=Rd,
                                                     vdim=LV, gate=og)
            put("latent_attention_expanded_prefill", f, flops=2.0 * pairs * LH * (LD + Rd + LV) + 2.0 * T * LH * (LD + LV) * Rk)
            f = lambda: ho.latent_attention_expanded(qp, plain, ws, wv, qs, ctx0, bt, sink, LH, LD, Rk, page, win, LD ** -0.5, 128, T, T, T, out=o)
            put("patadra_latent_attention_expanded_prefill", f, flops=2.0 * pairs * LH * (LD + LV) + 2.0 * T * LH * (LD + LV) * Rk)
            del wk, ws, q, qp, o
        else:
            ql = torch.randn((T, LH * R), device=dev) * 0.1
            qk = ql[:, :LH * Rk].contiguous()
            f = lambda: ho.latent_attention_paged(ql, cache, pos, tseq, bt, None, LH, R, page, win, R ** -0.5, n, query_start=qs, max_seq_len=ctx + n, out_cols=Rk)
            put("latent_attention_decode", f, nbytes=keys * R * 2, flops=2.0 * pairs * LH * (R + Rk))
            f = lambda: ho.latent_attention_paged(qk, plain, pos, tseq, bt, None, LH, Rk, page, win, R ** -0.5, n, query_start=qs, max_seq_len=ctx + n)
            put("patadra_latent_attention_decode", f, nbytes=keys * Rk * 2, flops=4.0 * pairs * LH * Rk)
            wv, ol = rn(LH * LV, Rk) * Rk ** -0.5, torch.randn((T, LH, R), device=dev)
            op = ol[:, :, :Rk].contiguous()
            nb = LH * LV * Rk * 2 + T * LH * Rk * 4 + T * LH * LV * 2
            put("latent_expand_values_gated_decode", lambda: ho.latent_expand_values(ol, wv, LH, LV, Rk, bf, gate=og), nbytes=nb + T * LH * LV * 2)
            put("patadra_head_project_decode", lambda: ho.head_project(op, wv, LH, LV, Rk, False), nbytes=nb)
        del cache, plain, og
        torch.cuda.empty_cache()
    # ---- the recurrent block ----
    C, nb, taps = d["width"], d["blocks"], d["taps"]
    n = C // nb
    wg, br, rate = rn(nb, 2 * n, n) * n ** -0.5, torch.zeros(C, device=dev), -torch.rand(C, device=dev)
    w1, ib = torch.randn((C, taps), device=dev), torch.randn(C, device=dev)
    for name, T, B in (("prefill", PROMPT, 1), ("decode", BATCH, BATCH)):
        qs = i32([i * (T // B) for i in range(B + 1)])
        tseq = torch.arange(B, device=dev, dtype=torch.int32).repeat_interleave(T // B)
        ctx, slots = i32([0 if name == "prefill" else CTX] * B), i32(list(range(B)))
        u, y = rn(T, C), rn(T, C)
        put(f"lru_gates_{name}", lambda: ho.lru_gates(u, wg, br, br, rate, nb), flops=4.0 * T * C * n, nbytes=T * C * (2 + 8) + 2 * C * n * 2)
        w2 = wg.reshape(nb * 2 * n, n)
        put(f"patadra_head_project_same_products_{name}", lambda: ho.head_project(u.reshape(T, nb, n), w2[: nb * n], nb, n, n, True), flops=2.0 * T * C * n,
            nbytes=T * C * (2 + 4) + C * n * 2)
        dec, inp = torch.rand((T, C), device=dev), torch.randn((T, C), device=dev)
        st = torch.zeros((B, C), device=dev)
        put(f"linear_scan_{name}", lambda: ho.linear_scan(dec, inp, y, br, st, slots, qs, ctx, T // B), nbytes=T * C * (8 + 2 + 2) + B * C * 8)
        zxg, b3 = rn(T, 3 * C), torch.zeros(3 * C, device=dev)
        put(f"lilovik_mingru_scan_{name}", lambda: ho.mingru_scan(zxg, b3, st, slots, qs, ctx, T // B), nbytes=T * C * (3 * 2 + 2) + B * C * 8)
        hist = torch.zeros((B, (taps - 1) * C), device=dev)
        put(f"short_filter_{name}", lambda: ho.tap_filter(u, w1, None, hist, slots, tseq, qs, ctx, False, 0, in_bias=ib, bias1=ib), nbytes=T * C * 4 + B * (taps - 1) * C * 8)
        put(f"surinex_tap_filter_{name}", lambda: ho.tap_filter(u, w1, None, hist, slots, tseq, qs, ctx, False, 1), nbytes=T * C * 4 + B * (taps - 1) * C * 8)
        del zxg, dec, inp
    # ---- row operators at 8192 tokens ----
    T = 8192
    x, y, wn = torch.randn((T, W), device=dev), rn(T, W), torch.ones(W, device=dev)
    put("postnorm_residual", lambda: ho.postnorm_residual(x, wn, 2.0, 1e-5, bf, y=y), nbytes=T * W * (8 + 2 + 2))
    for nd in (2, 4, 16):
        depth, dw = torch.randn((nd, T, W), device=dev), torch.full((nd,), 1.0 / nd, device=dev)
        put(f"postnorm_residual_depth_{nd}", lambda: ho.postnorm_residual(x, wn, 2.0, 1e-5, bf, y=y, depth=depth, depth_w=dw, depth_n=nd), nbytes=T * W * (8 + 2 + 2 + 4 * nd))
        del depth
    x4, mix, w4 = torch.randn((T, 4, W), device=dev), torch.eye(4, device=dev), torch.ones(4, device=dev)
    put("nemasun_lanes_update_norm", lambda: ho.lanes_update_norm(x4, y, mix, w4, bf, eps=1e-6, w_in_next=w4, w_next=wn), nbytes=T * W * (2 + 32 + 2))
    put("lilovik_postnorm_add_prenorm", lambda: ho.postnorm_add_prenorm(y, x, wn, wn, 1e-5, 0.0), nbytes=T * W * (2 + 8 + 2))
    del x, x4, y
    N = H * D + 2 * G * D
    proj, pos, slot = rn(T, N), torch.arange(T, device=dev), torch.randperm(T, device=dev)
    kc, vc = torch.empty((T, G, D), device=dev, dtype=bf), torch.empty((T, G, D), device=dev, dtype=bf)
    bias, hs, qw = torch.randn(N, device=dev), torch.ones(H, device=dev), torch.ones(D, device=dev)
    put("qkv_unitnorm_bias_cache", lambda: ho.qkv_headnorm_rope_cache(proj, 0, H * D, H * D + G * D, None, None, None, None, False, pos, slot, kc, vc, H, G, D, D, 1e-5,
                                                                     bias=bias, q_head_scale=hs, unit_norm=True), nbytes=T * 2 * (2 * N))
    put("nemasun_qk_headnorm_cache", lambda: ho.qk_headnorm_cache(proj, 0, H * D, H * D + G * D, qw, qw, 0.0, slot, kc, vc, H, G, D, D, 1e-6), nbytes=T * 2 * (2 * N))
    Rq = l["q_rank"]
    proj = rn(T, Rq + R)
    cache, freq = torch.empty((T, R), device=dev, dtype=bf), torch.rand(Rd // 2, device=dev)
    plain = torch.empty((T, Rk), device=dev, dtype=bf)
    qn, kn = torch.ones(Rq, device=dev), torch.ones(Rk, device=dev)
    put("latent_norm_rope_cache", lambda: ho.latent_norm_rope_cache(proj, qn, kn, freq, True, pos, slot, cache, Rq, Rk, Rd, 1e-5, freq_lo=freq, amplitude=1.2), nbytes=T * (Rq + R) * 4)
    put("patadra_latent_norm_cache", lambda: ho.latent_norm_cache(proj, qn, kn, slot, plain, Rq, Rk, 1e-5), nbytes=T * (Rq + Rk) * 4)
    del proj, cache, plain, kc, vc
    torch.cuda.empty_cache()
    # ---- router and routed experts ----
    E, top, ff = s["experts"], s["top"], s["expert_ff"]
    wgu, wd = rn(E, 2 * ff, W) * W ** -0.5, rn(E, W, ff) * ff ** -0.5
    wr, corr = torch.randn((E, W), device=dev) * W ** -0.5, torch.randn(E, device=dev) * 0.01
    for name, T in (("prefill", PROMPT), ("decode", BATCH)):
        h = rn(T, W)
        idx, wgt = ho.moe_route_grouped(h, wr, corr, top, s["groups"], s["keep_groups"], score="sigmoid", group_top=2)
        used = int(torch.unique(idx).numel())
        put(f"experts_{name}", lambda: ho.moe_expert_rows(h, idx, wgt, wgu, wd, 0.0, 1.0, 0.0, scale_input=False), flops=6.0 * T * top * ff * W, nbytes=used * 3 * ff * W * 2)
        put(f"router_{name}", lambda: ho.moe_route_grouped(h, wr, corr, top, s["groups"], s["keep_groups"], score="sigmoid", group_top=2), nbytes=T * W * 2 + E * W * 4)
        put(f"nemasun_router_{name}", lambda: ho.moe_route_grouped(h, wr, corr, top, s["groups"], s["keep_groups"]), nbytes=T * W * 2 + E * W * 4)
    return rows


def run(args, torch, dev, json_fd):
    from atoma_infer_b200 import _lib
    from bench import ClockSampler
    if args.impl != "ours":
        os.write(json_fd, (json.dumps({"impl": "reference", "unavailable": "the reference has no model of this design"}) + "\n").encode())
        return
    _lib.lib()
    hbm, tf, src = _peaks()
    steps, warmup = max(1, args.steps), max(3, args.warmup)
    out_sizes, headline = {}, None
    sampler, t_clock0 = ClockSampler(torch.cuda.current_device()), time.time()
    for name, s in SIZES.items():
        spec = _spec(s)
        mine = _serve(torch, spec, _weights(torch, spec, s, dev), dev, steps, warmup)
        ns = _nemasun_sizes(s)
        nspec = bench_nemasun._spec(ns)
        nemasun = _serve(torch, nspec, bench_nemasun._weights(torch, nspec, ns, dev), dev, steps, warmup)
        rows = _kernel_rows(torch, s, dev, max(3, steps // 2), 3, hbm, tf)
        torch.cuda.empty_cache()
        out_sizes[name] = {"sizes": {k: (list(v) if isinstance(v, tuple) else v) for k, v in s.items()}, **mine, "nemasun_equal_size": nemasun, "kernels": rows}
        headline = out_sizes[name]
    clocks = sampler.stop(t_clock0, time.time())
    h2d = BATCH * (4 + 8 + 8 + 4 + 4 + 4 + 4) + BATCH * ((CTX + 64) // 16 + 1) * 4
    line = {
        "metric": "Mobunex decode tokens/s, batch 32, context 4096, 4k-wide layer sizes (3 layers), through the engine's executor",
        "value": headline["decode_graph_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup,
        "ms_per_step": headline["decode_graph_ms_per_step"], "higher_is_better": True, "scaling": "strong", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic (random weights, random tokens)", "impl": "ours", "gpu_launches": headline["decode_launches_per_step"],
        "clocks": clocks,
        "e2e": {"value": headline["decode_tokens_per_s"], "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": BATCH * 4},
        "config": {"design": "Mobunex", "batch": BATCH, "ctx": CTX, "prompt": PROMPT, "peaks": src, "hbm_gbs": hbm, "bf16_tflops": tf,
                   "l2": "kernel rows flush L2 between iterations; model steps stream more than L2", "sizes": out_sizes},
    }
    os.write(json_fd, (json.dumps(line) + "\n").encode())
