"""bench.py --design lusalorn: prefill and decode throughput of the Lusalorn design (random weights) at sizes that resemble real models'
layers, beside the framework's closest existing model — Surinex, whose pair of mixers (attention beside a gated delta rule with the same
heads and state) is the nearest to this design's sum of attention and a state-space recurrence — at equal width, head counts, head sizes,
state, feed-forward size and number of layers, and the design's own kernels against the measured peaks beside the like kernels of the
models they come from (Surinex's scan, filter, head norm and rotation, Mobunex's softmax attention and post-norm update).  Not the headline
(config 2 is); ONE JSON line in the same format.

Per size: `prefill` = one 4096-token prompt in one step; `decode` = one step of 32 sequences at context 4096 (built by prefilling them),
timed with CUDA events around K executor steps after W warm-up steps, inputs shipped from pinned memory every step, sampled tokens read
back; the same step replayed from a CUDA graph is the device-only figure.  Kernel rows: achieved bytes/s or FLOP/s over the measured peaks
of MEASURED_PEAKS.json (fallback figures when absent); L2 is flushed between their iterations."""
from __future__ import annotations

import json
import math
import os
import time

import bench_surinex
from bench_hybrid import BATCH, CTX, PROMPT, _peaks, _time
from bench_mobunex import _serve
from bench_patadra import _row

SIZES = {
    "2k-wide": dict(width=2048, vocab=32000, ff=8192, window=1024, mult=0.9, attention=dict(heads=16, kv_heads=4, dim=64, vdim=128, rot=32),
                    left=dict(heads=32, kv_heads=8, dim=64, vdim=64, rot=64), right=dict(heads=32, vdim=64, groups=8, state=128, norm_groups=8, taps=4),
                    layers=("parallel", "attention", "parallel", "shared")),
    "4k-wide": dict(width=4096, vocab=32000, ff=14336, window=4096, mult=0.9, attention=dict(heads=32, kv_heads=8, dim=64, vdim=128, rot=32),
                    left=dict(heads=32, kv_heads=8, dim=128, vdim=128, rot=128), right=dict(heads=64, vdim=64, groups=8, state=128, norm_groups=8, taps=4),
                    layers=("parallel", "attention", "parallel", "shared")),
}


def _spec(s):
    from atoma_infer_b200.hybrid import (HybridSpec, LayerSpec, MixerSumSpec, MlpSpec, PairTableSpec, RotarySpec, SoftmaxAttentionSpec, StateSpaceSpec)
    a, l, d = s["attention"], s["left"], s["right"]
    source = s["layers"].index("attention")
    attn = lambda kv_from: dict(mixer="softmax_attention",
                                softmax=SoftmaxAttentionSpec(a["heads"], a["kv_heads"], a["dim"], a["vdim"], 1 / math.sqrt(a["dim"]), s["window"], bias=True, qk_norm=True,
                                                             rotary=RotarySpec(a["rot"], 1e5), out_bias=True, maps=2, diff=0.4, kv_from=kv_from))
    both = MixerSumSpec(SoftmaxAttentionSpec(l["heads"], l["kv_heads"], l["dim"], l["vdim"], 1 / math.sqrt(l["dim"]), qk_norm=True,
                                             rotary=RotarySpec(l["rot"], 5e5, yarn=(4.0, 2048, 32.0, 1.0))),
                        StateSpaceSpec(d["heads"], d["vdim"], d["groups"], d["state"], d["norm_groups"], d["taps"]), 0.8, 1.25)
    mixers = {"attention": attn(None), "shared": attn(source), "parallel": dict(mixer="attention_ssm", mixer_sum=both)}
    return HybridSpec(s["width"], s["vocab"], 1e-5, 1.0, tuple(LayerSpec(mlp=MlpSpec(s["ff"], "silu"), **mixers[k]) for k in s["layers"]), norm_offset=1.0,
                      block_style="postnorm", position="none", embed_norm=False, branch_scale=s["mult"], pair_table=PairTableSpec(30011, 1019, 31))


def _weights(torch, spec, s, dev):
    gen = torch.Generator(device=dev).manual_seed(23)

    def r(*shape, scale=1.0, mean=0.0):
        return (mean + torch.randn(shape, generator=gen, device=dev, dtype=torch.float32) * scale).to(torch.bfloat16)

    W, F = spec.width, s["ff"]
    lin = lambda o, i: r(o, i, scale=i ** -0.5)
    out = {"embed": r(spec.vocab, W), "pair_table": r(spec.pair_table.buckets + 1, W), "head": lin(spec.vocab, W), "final_norm": r(W, scale=0.1), "layers": []}
    for ls in spec.layers:
        w = {"norm1": r(W, scale=0.1), "norm2": r(W, scale=0.1), "w_gate_up": lin(2 * F, W), "w_down": lin(W, F)}
        a = ls.softmax if ls.softmax is not None else ls.mixer_sum.left
        M = a.maps
        w.update(w_q=lin(M * a.heads * a.dim, W), q_norm=r(a.dim, scale=0.1, mean=1.0), w_o=lin(W, a.heads * a.vdim))
        if a.kv_from is None:
            w.update(w_k=lin(M * a.kv_heads * a.dim, W), w_v=lin(a.kv_heads * a.vdim, W), k_norm=r(a.dim, scale=0.1, mean=1.0))
        if a.bias:
            w.update(b_q=r(M * a.heads * a.dim, scale=0.1), b_k=r(M * a.kv_heads * a.dim, scale=0.1), b_v=r(a.kv_heads * a.vdim, scale=0.1), b_o=r(W, scale=0.1),
                     diff_lambda=0.4)
        if ls.mixer_sum is not None:
            d = ls.mixer_sum.right
            w.update(r_w_z=lin(d.inner, W), r_w_x=lin(d.inner, W), r_w_bc=lin(2 * d.groups * d.state, W), r_w_dt=lin(d.heads, W),
                     r_tap_w=r(d.channels, d.taps, scale=0.5), r_tap_b=r(d.channels, scale=0.1), r_dt_bias=r(d.heads, mean=-2.0), r_a_log=r(d.heads),
                     r_skip=r(d.heads), r_norm=r(d.inner, scale=0.1, mean=1.0), r_w_o=lin(W, d.inner))
        out["layers"].append(w)
    return out


def _surinex_spec(s):
    """A Surinex model of pair layers only, of equal width, heads, head sizes, state, feed-forward size and number of layers."""
    from atoma_infer_b200.hybrid import DeltaRuleSpec, HybridSpec, LayerSpec, MixerPairSpec, MlpSpec, RotarySigmoidAttentionSpec, RotarySpec
    l, d = s["left"], s["right"]
    pair = MixerPairSpec(RotarySigmoidAttentionSpec(l["heads"], l["kv_heads"], l["dim"], l["vdim"], 1 / math.sqrt(l["dim"]), RotarySpec(l["rot"], 1e6, True)),
                         DeltaRuleSpec(d["heads"], d["groups"], d["state"], d["vdim"], d["taps"]))
    layers = tuple(LayerSpec(mixer="pair", pair=pair, mlp=MlpSpec(s["ff"], "silu"), source=i, taps=4) for i in range(len(s["layers"])))
    return HybridSpec(s["width"], s["vocab"], 1e-5, 1.0, layers, norm_offset=0.0, block_style="parallel", position="none")


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

    a, l, d = s["attention"], s["left"], s["right"]
    H, G, D, V = 2 * a["heads"], 2 * a["kv_heads"], a["dim"], a["vdim"]
    # ---- attention: one 4096-token prompt, and a decode step of BATCH sequences at context CTX ----
    for name, T, B, ctx in (("prefill", PROMPT, 1, 0), ("decode", BATCH, BATCH, CTX)):
        n = T // B
        mb = (ctx + n + page - 1) // page
        bt = torch.randperm(B * mb, device=dev).to(torch.int32).reshape(B, mb)
        pos = (torch.arange(n, device=dev) + ctx).repeat(B)
        tseq, qs = torch.arange(B, device=dev, dtype=torch.int32).repeat_interleave(n), i32([i * n for i in range(B + 1)])
        kw = dict(max_query_len=n, query_start=qs, max_seq_len=ctx + n)
        if name == "prefill":
            kw.update(long_min_q=128, long_stats=(1, T, 0))

        def attention(key, H, G, share, D, V, window):
            pairs = B * sum(min(ctx + i + 1, window or (1 << 30)) for i in range(n))
            keys = B * min(ctx + n, (window or (1 << 30)) + n - 1)
            kc, vc, q = rn(B * mb * page, G, D), rn(B * mb * page, G // share, V), rn(T, H * D)
            out = torch.empty((T, H * V), device=dev, dtype=bf)
            put(f"{key}_{name}", lambda: ho.softmax_attention_paged(q, kc, vc, pos, tseq, bt, H, G, D, V, page, D ** -0.5, window=window, out=out, v_share=share, **kw),
                flops=2.0 * pairs * H * (D + V), nbytes=keys * (G * D + G // share * V) * 2)

        attention("differential_maps", H, G, 2, D, V, win)
        attention("mobunex_softmax_attention", H, G, 1, D, D, win)                       # as many heads, values as long as keys
        attention("mobunex_softmax_attention_128", H // 2, G // 2, 1, V, V, win)          # as many value bytes
        attention("left_attention", l["heads"], l["kv_heads"], 1, l["dim"], l["vdim"], 0)
        maps = rn(T, H * V)
        put(f"differential_combine_{name}", lambda: ho.differential_combine(maps, H // 2, G // 2, V, 0.4, 0.6, 1e-5), nbytes=T * H * V * 3)
        del maps
        torch.cuda.empty_cache()
        # ---- the recurrence beside the attention ----
        RH, RG, N, P = d["heads"], d["groups"], d["state"], d["vdim"]
        inner, C = RH * P, RH * P + 2 * RG * N
        ctxs, slots = i32([ctx] * B), i32(list(range(B)))
        conv, dt, z = rn(T, C), rn(T, RH), rn(T, inner)
        h1 = torch.zeros(RH, device=dev)
        st = torch.zeros((B, RH * N * P), device=dev)
        x_, b_, c_ = conv[:, :inner], conv[:, inner:inner + RG * N], conv[:, inner + RG * N:]
        sb = T * C * 2 + T * inner * 4 + B * RH * N * P * 8
        put(f"ssm_scan_{name}", lambda: ho.ssm_scan(x_, b_, c_, dt, h1, h1, h1, st, slots, qs, ctxs, RH, RG, N, P), nbytes=sb, flops=5.0 * T * RH * N * P)
        put(f"surinex_delta_scan_{name}", lambda: ho.delta_rule_scan(c_, b_, x_, dt, dt, h1, h1, 1.0, st, slots, qs, ctxs, RH, RG, N, P), nbytes=sb, flops=7.0 * T * RH * N * P)
        k2, v2, z2 = rn(T, RH * N), rn(T, RH * P), rn(T, RH * N)
        zb = torch.zeros(RH * N, device=dev)
        put(f"surinex_gla_scan_{name}", lambda: ho.gla_scan(k2, k2, v2, z2, zb, 16.0, 1.0, st, slots, qs, ctxs, RH, N, P),
            nbytes=T * (3 * RH * N + inner) * 2 + T * inner * 4 + B * RH * N * P * 8, flops=5.0 * T * RH * N * P)
        del k2, v2, z2
        o = torch.randn((T, inner), device=dev)
        wn, hn = torch.ones(inner, device=dev), torch.ones(P, device=dev)
        put(f"gate_groupnorm_{name}", lambda: ho.gate_groupnorm(o, z, wn, d["norm_groups"], 1e-5), nbytes=T * inner * 8)
        put(f"surinex_headnorm_gate_{name}", lambda: ho.headnorm_gate(o, hn, z, RH, P, 1e-5, bf), nbytes=T * inner * 8)
        w1, b1, hist = torch.randn((C, d["taps"]), device=dev), torch.randn(C, device=dev), torch.zeros((B, (d["taps"] - 1) * C), device=dev)
        nb = T * C * 4 + B * (d["taps"] - 1) * C * 8
        put(f"short_filter_{name}", lambda: ho.tap_filter(conv, w1, None, hist, slots, tseq, qs, ctxs, False, 1, bias1=b1), nbytes=nb)
        put(f"surinex_tap_filter_{name}", lambda: ho.tap_filter(conv, w1, None, hist, slots, tseq, qs, ctxs, False, 1), nbytes=nb)
        del conv, dt, z, o, st, hist
        torch.cuda.empty_cache()
    # ---- row operators at 8192 tokens ----
    T = 8192
    x, y, wn = torch.randn((T, W), device=dev), rn(T, W), torch.ones(W, device=dev)
    put("branch_norm_update", lambda: ho.postnorm_residual(x, wn, 1.0, 1e-5, bf, y=y, offset=1.0, branch_scale=0.9, y_bias=wn), nbytes=T * W * (8 + 2 + 2))
    put("mobunex_postnorm_residual", lambda: ho.postnorm_residual(x, wn, 2.0, 1e-5, bf, y=y), nbytes=T * W * (8 + 2 + 2))
    toks, tseq, qs = torch.randint(0, s["vocab"], (T,), device=dev, dtype=torch.int32), torch.zeros(T, device=dev, dtype=torch.int32), i32([0, T])
    table, pairs = rn(s["vocab"], W), rn(30012, W)
    put("embed_pairs", lambda: ho.embed_pairs(toks, tseq, qs, i32([-1]), table, pairs, 30011, 1019, 31), nbytes=T * W * (2 + 2 + 4 + 2))
    put("mobunex_embedding", lambda: ho.embed_scaled_lanes(toks, table, 1.0, 1), nbytes=T * W * (2 + 4))
    del x, y, table, pairs
    pos, slot = torch.arange(T, device=dev), torch.randperm(T, device=dev)
    for key, H, G, Gv, D, V, rot in (("differential", 2 * a["heads"], 2 * a["kv_heads"], a["kv_heads"], a["dim"], a["vdim"], a["rot"]),
                                     ("left", l["heads"], l["kv_heads"], l["kv_heads"], l["dim"], l["vdim"], l["rot"])):
        N = H * D + G * D + Gv * V
        proj = rn(T, N)
        kc, vc = torch.empty((T, G, D), device=dev, dtype=bf), torch.empty((T, Gv, V), device=dev, dtype=bf)
        bias, qw, f = torch.randn(N, device=dev), torch.ones(D, device=dev), torch.rand(rot // 2, device=dev)
        put(f"qkv_norm_rope_cache_{key}", lambda: ho.qkv_headnorm_rope_cache(proj, 0, H * D, H * D + G * D, qw, qw, f, None, False, pos, slot, kc, vc, H, G, D, V, 1e-5,
                                                                             bias=bias if key == "differential" else None, qk_freq_lo=f, amplitude=1.1, v_heads=Gv),
            nbytes=T * 2 * (2 * N))
        if key == "left":
            fv = torch.rand(V // 2, device=dev)
            put("surinex_qkv_headnorm_rope_cache", lambda: ho.qkv_headnorm_rope_cache(proj, 0, H * D, H * D + G * D, qw, qw, f, fv, False, pos, slot, kc, vc, H, G, D, V,
                                                                                      1e-5), nbytes=T * 2 * (2 * N))
            put("nemasun_qk_headnorm_cache", lambda: ho.qk_headnorm_cache(proj, 0, H * D, H * D + G * D, qw, qw, 0.0, slot, kc, vc, H, G, D, V, 1e-6), nbytes=T * 2 * (2 * N))
        del proj, kc, vc
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
        sspec = _surinex_spec(s)
        surinex = _serve(torch, sspec, bench_surinex._weights(torch, sspec, dict(ff=s["ff"], taps=4), dev), dev, steps, warmup)
        rows = _kernel_rows(torch, s, dev, max(3, steps // 2), 3, hbm, tf)
        torch.cuda.empty_cache()
        out_sizes[name] = {"sizes": {k: (list(v) if isinstance(v, tuple) else v) for k, v in s.items()}, **mine, "surinex_equal_size": surinex, "kernels": rows}
        headline = out_sizes[name]
    clocks = sampler.stop(t_clock0, time.time())
    h2d = BATCH * (4 + 8 + 8 + 4 + 4 + 4 + 4 + 4) + BATCH * ((CTX + 64) // 16 + 1) * 4
    line = {
        "metric": "Lusalorn decode tokens/s, batch 32, context 4096, 4k-wide layer sizes (4 layers), through the engine's executor",
        "value": headline["decode_graph_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup,
        "ms_per_step": headline["decode_graph_ms_per_step"], "higher_is_better": True, "scaling": "strong", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic (random weights, random tokens)", "impl": "ours", "gpu_launches": headline["decode_launches_per_step"],
        "clocks": clocks,
        "e2e": {"value": headline["decode_tokens_per_s"], "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": BATCH * 4},
        "config": {"design": "Lusalorn", "batch": BATCH, "ctx": CTX, "prompt": PROMPT, "peaks": src, "hbm_gbs": hbm, "bf16_tflops": tf,
                   "l2": "kernel rows flush L2 between iterations; model steps stream more than L2", "sizes": out_sizes},
    }
    os.write(json_fd, (json.dumps(line) + "\n").encode())
