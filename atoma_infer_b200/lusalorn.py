"""Lusalorn: a decoder whose sublayers' results are normed before they join the stream, with differential attention under a sliding window
(some layers on an earlier layer's keys and values) and layers that sum softmax attention and a state-space recurrence.

config.json gives every size and every constant that can differ between checkpoints:
  architecture "Lusalorn", vocab, width, norm {eps}, residual_mult (factor of a sublayer's normed result), embedding {bigram {buckets, mul_prev,
  mul_cur}}, and `layers`: per layer its `type` ("attention" | "parallel"), the mixer's sizes (`mixer`) and its feed-forward (`mlp`
  {kind "dense", ff}, null for none).
    attention:  heads, kv_heads, dim, vdim, scale, diff, rot {base, dims}, mask {size}, kv_from? (the layer whose keys and values are used)
    parallel:   left {heads, kv_heads, dim, vdim, scale, rot {base, dims, scaling {factor, original, fast, slow}}},
                right {heads, vdim, groups, state, norm_groups, conv}, left_scale, right_scale
Fixed by the design (and therefore constants here): norm weights are stored around zero; x <- x + m norm1(mixer(x)), x <- x + m norm2(ff(x));
q and k are RMS-normed per head with a plain weight before the rotation, which pairs (i, i + dims / 2).  Attention: two softmax maps per
head over the same values, o = a1 - lambda a2 at unit root mean square times 1 - diff, lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff;
biases on all four projections.  Parallel: causal softmax attention without biases beside a state-space recurrence with a scalar decay per
head.  Feed-forward: W_down (silu(W_gate h) * W_up h).

Checkpoint tensors: embed, bigram [buckets + 1, width], head, final.norm, and per layer i `l<i>.norm1`, `l<i>.norm2` (with a feed-forward),
`l<i>.mlp.{gate, up, down}`, and under `l<i>.mix.`:
    attention:  q, q.b, q.norm, lq1, lk1, lq2, lk2, o, o.b, and without kv_from k, k.b, k.norm, v, v.b
                (a head's rows of q and k are [map 1, map 2])
    parallel:   left.{q, k, v, q.norm, k.norm, o}, right.{in, conv, conv.b, dt_bias, A_log, D, norm, o}   (rows of in: z, x, B, C, dt)
This module turns that into the generic hybrid description (hybrid.py); it has no compute of its own.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .hybrid import (HybridSpec, LayerSpec, MixerSumSpec, MlpSpec, PairTableSpec, RotarySpec, SoftmaxAttentionSpec, StateSpaceSpec)
from .ops import AtomaError

ARCHITECTURE = "Lusalorn"


def _window(m: dict) -> int:
    mask = m.get("mask")
    if not mask or mask.get("size") is None:
        return 0
    size = int(mask["size"])
    if size < 1:
        raise AtomaError(f"a window of {size} tokens")
    return size


def _rotary(rot: Optional[dict]) -> Optional[RotarySpec]:
    if not rot or int(rot["dims"]) == 0:
        return None
    sc = rot.get("scaling")
    yarn = None if not sc else (float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"]))
    return RotarySpec(dims=int(rot["dims"]), base=float(rot["base"]), yarn=yarn)


def _heads(m: dict) -> dict:
    return dict(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                qk_norm=True, rotary=_rotary(m.get("rot")), window=_window(m))


def _layer_spec(i: int, l: dict) -> LayerSpec:
    kind, m, f = l.get("type"), l["mixer"], l.get("mlp")
    if f is not None and f.get("kind", "dense") != "dense":
        raise AtomaError(f"layer {i}: feed-forward kind {f['kind']!r} is not part of the Lusalorn design")
    ff = {} if f is None else dict(mlp=MlpSpec(ff=int(f["ff"]), act="silu"))
    if kind == "attention":
        kv_from = m.get("kv_from")
        return LayerSpec("softmax_attention", softmax=SoftmaxAttentionSpec(**_heads(m), bias=True, out_bias=True, maps=2, diff=float(m["diff"]),
                                                                           kv_from=None if kv_from is None else int(kv_from)), **ff)
    if kind == "parallel":
        r = m["right"]
        right = StateSpaceSpec(heads=int(r["heads"]), vdim=int(r["vdim"]), groups=int(r["groups"]), state=int(r["state"]),
                               norm_groups=int(r["norm_groups"]), taps=int(r["conv"]))
        return LayerSpec("attention_ssm", mixer_sum=MixerSumSpec(SoftmaxAttentionSpec(**_heads(m["left"])), right, float(m["left_scale"]),
                                                                 float(m["right_scale"])), **ff)
    raise AtomaError(f"layer {i}: mixer type {kind!r} is not part of the Lusalorn design")


def spec_from_config(cfg: dict) -> HybridSpec:
    big = (cfg.get("embedding") or {}).get("bigram")
    pair = None if not big else PairTableSpec(int(big["buckets"]), int(big["mul_prev"]), int(big["mul_cur"]))
    return HybridSpec(width=int(cfg["width"]), vocab=int(cfg["vocab"]), eps=float(cfg["norm"]["eps"]), logit_scale=1.0,
                      layers=tuple(_layer_spec(i, l) for i, l in enumerate(cfg["layers"])), norm_offset=1.0, block_style="postnorm", position="none",
                      embed_norm=False, branch_scale=float(cfg["residual_mult"]), pair_table=pair)


def weights_from_checkpoint(spec: HybridSpec, ckpt: Dict[str, torch.Tensor]) -> dict:
    """Checkpoint names -> the generic hybrid layout."""
    W = spec.width

    def get(name, shape):
        if name not in ckpt:
            raise AtomaError(f"tensor {name} is missing from the checkpoint")
        t = ckpt[name]
        if tuple(t.shape) != tuple(shape):
            raise AtomaError(f"tensor {name} has shape {tuple(t.shape)}, the configuration needs {tuple(shape)}")
        return t

    out = {"embed": get("embed", (spec.vocab, W)), "head": get("head", (spec.vocab, W)), "final_norm": get("final.norm", (W,)), "layers": []}
    if spec.pair_table is not None:
        out["pair_table"] = get("bigram", (spec.pair_table.buckets + 1, W))
    for i, ls in enumerate(spec.layers):
        p, q = f"l{i}.", f"l{i}.mix."
        w = {"norm1": get(p + "norm1", (W,))}
        if ls.softmax is not None:
            a = ls.softmax
            nq, nk, nv = 2 * a.heads * a.dim, 2 * a.kv_heads * a.dim, a.kv_heads * a.vdim
            w.update(w_q=get(q + "q", (nq, W)), b_q=get(q + "q.b", (nq,)), q_norm=get(q + "q.norm", (a.dim,)), w_o=get(q + "o", (W, a.heads * a.vdim)),
                     b_o=get(q + "o.b", (W,)))
            if a.kv_from is None:
                w.update(w_k=get(q + "k", (nk, W)), b_k=get(q + "k.b", (nk,)), k_norm=get(q + "k.norm", (a.dim,)), w_v=get(q + "v", (nv, W)),
                         b_v=get(q + "v.b", (nv,)))
            lq1, lk1, lq2, lk2 = (get(q + n, (a.dim,)).double() for n in ("lq1", "lk1", "lq2", "lk2"))
            w["diff_lambda"] = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum())) + a.diff
        else:
            a, d = ls.mixer_sum.left, ls.mixer_sum.right
            l, r = q + "left.", q + "right."
            w.update(w_q=get(l + "q", (a.heads * a.dim, W)), w_k=get(l + "k", (a.kv_heads * a.dim, W)), w_v=get(l + "v", (a.kv_heads * a.vdim, W)),
                     q_norm=get(l + "q.norm", (a.dim,)), k_norm=get(l + "k.norm", (a.dim,)), w_o=get(l + "o", (W, a.heads * a.vdim)))
            rows = get(r + "in", (d.inner + d.channels + d.heads, W))
            w["r_w_z"], w["r_w_x"], w["r_w_bc"], w["r_w_dt"] = torch.split(rows, [d.inner, d.inner, 2 * d.groups * d.state, d.heads], 0)
            w.update(r_tap_w=get(r + "conv", (d.channels, d.taps)), r_tap_b=get(r + "conv.b", (d.channels,)), r_dt_bias=get(r + "dt_bias", (d.heads,)),
                     r_a_log=get(r + "A_log", (d.heads,)), r_skip=get(r + "D", (d.heads,)), r_norm=get(r + "norm", (d.inner,)),
                     r_w_o=get(r + "o", (W, d.inner)))
        if ls.mlp is not None:
            f, n = p + "mlp.", ls.mlp.ff
            w["norm2"] = get(p + "norm2", (W,))
            w["w_gate_up"] = torch.cat([get(f + "gate", (n, W)), get(f + "up", (n, W))], 0)
            w["w_down"] = get(f + "down", (W, n))
        out["layers"].append(w)
    return out
