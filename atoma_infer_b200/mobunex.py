"""Mobunex: a decoder of post-norm blocks with an average over depth, whose layers mix windowed softmax attention, windowed latent
attention and a recurrent block, with dense or routed feed-forwards.

config.json gives every size and every constant that can differ between checkpoints:
  architecture "Mobunex", vocab, width, norm {eps}, postln_alpha (the stream's factor in every sum), and `layers`: per layer its `type`
  ("attention" | "latent_attention" | "rglru"), the mixer's sizes (`mixer`) and its feed-forward (`mlp`, null for none).
    attention:         heads, kv_heads, dim, vdim, scale, mask {size}
    latent_attention:  heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mask {size}, rot {base, dims, scaling? {factor, original, fast, slow}}
    rglru:             width, blocks, conv
    mlp:               {kind "dense", ff} or {kind "moe", expert {ff}, router {experts, top, groups? {count, keep}}, shared? {ff}}
Fixed by the design (and therefore constants here): a norm's weight is one number for all coordinates; the embedding rows are normed;
x <- norm1(alpha x + mixer(x)), x <- norm2(alpha x + ff(x)), and a layer hands on a weighted sum of the embedding output and of all
results so far.  Attention: projection biases, q and k divided by their root mean square per head, a factor per head on the score, no
positions.  Latent attention: normed query and key/value latents, heads laid out [dim plain | rot_dim rotated], one rotated key part for
all heads, pairs (2i, 2i + 1) with YaRN scaling, a sigmoid gate on the heads' outputs.  Recurrent block: a gate branch through gelu, a
branch through a causal filter with bias and the unit log a = -8 r softplus(lam), S <- a S + sqrt(1 - a^2) i u.  Router: sigmoid scores,
the choice corrected and restricted to the groups with the largest sums of two choice scores, weights renormalised, on the experts'
outputs.  Feed-forwards: W_down (silu(W_gate h) * W_up h).

Checkpoint tensors: embed, embed.norm, head, final.norm, and per layer i `l<i>.norm1`, `l<i>.norm2` (with a feed-forward), `l<i>.dwa` [i + 2],
`l<i>.mlp.{gate, up, down}` or `l<i>.mlp.{router, correction}`, `l<i>.mlp.e<k>.{gate, up, down}`, `l<i>.mlp.shared.{gate, up, down}`, and under
`l<i>.mix.`:
    attention:         q, k, v (each with .b), temp, o
    latent_attention:  dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o
    rglru:             y, x (each with .b), conv, conv.b, ra, ra.b, ri, ri.b, lam, o
This module turns that into the generic hybrid description (hybrid.py); it has no compute of its own.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .hybrid import (HybridSpec, LatentAttentionSpec, LayerSpec, LinearRecurrentSpec, MlpSpec, MoeSpec, RotarySpec, SoftmaxAttentionSpec)
from .ops import AtomaError

ARCHITECTURE = "Mobunex"
DECAY_FACTOR = 8.0          # log a = -8 r softplus(lam)


def _window(m: dict) -> int:
    mask = m.get("mask")
    if not mask:
        return 0
    size = int(mask["size"])
    if size < 1:
        raise AtomaError(f"a window of {size} tokens")
    return size


def _rotary(rot: Optional[dict], rot_dim: int) -> Optional[RotarySpec]:
    if rot_dim == 0:
        return None
    rot = rot or {}
    sc = rot.get("scaling")
    yarn = None if not sc else (float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"]))
    return RotarySpec(dims=int(rot.get("dims", rot_dim)), base=float(rot.get("base", 10000.0)), interleaved=True, yarn=yarn)


def _feed_forward(i: int, f: Optional[dict]) -> dict:
    if f is None:
        return {}
    kind = f.get("kind", "dense")
    if kind == "dense":
        return dict(mlp=MlpSpec(ff=int(f["ff"]), act="silu"))
    if kind != "moe":
        raise AtomaError(f"layer {i}: feed-forward kind {kind!r} is not part of the Mobunex design")
    r, groups, shared = f["router"], f["router"].get("groups"), f.get("shared")
    return dict(moe=MoeSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(f["expert"]["ff"]), shared_ff=int(shared["ff"]) if shared else 0,
                            alpha=1.0, up_shift=0.0, renormalize=True, score="sigmoid", correction=True,
                            groups=int(groups["count"]) if groups else 1, keep_groups=int(groups["keep"]) if groups else 1, group_top=2,
                            scale_input=False))


def _layer_spec(i: int, l: dict) -> LayerSpec:
    kind, m = l.get("type"), l["mixer"]
    ff = _feed_forward(i, l.get("mlp"))
    if kind == "attention":
        return LayerSpec("softmax_attention",
                         softmax=SoftmaxAttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                                      scale=float(m["scale"]), window=_window(m), bias=True, head_scale=True), **ff)
    if kind == "latent_attention":
        rot_dim = int(m.get("rot_dim", 0))
        return LayerSpec("latent_attention",
                         latent=LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), q_rank=int(m["q_rank"]),
                                                    kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), window=_window(m), rot_dim=rot_dim,
                                                    rotary=_rotary(m.get("rot"), rot_dim), out_gate=True), **ff)
    if kind == "rglru":
        return LayerSpec("lru", lru=LinearRecurrentSpec(width=int(m["width"]), blocks=int(m["blocks"]), taps=int(m["conv"]), act="gelu_tanh"), **ff)
    raise AtomaError(f"layer {i}: mixer type {kind!r} is not part of the Mobunex design")


def spec_from_config(cfg: dict) -> HybridSpec:
    norm = cfg.get("norm") or {}
    return HybridSpec(width=int(cfg["width"]), vocab=int(cfg["vocab"]), eps=float(norm.get("eps", 1e-6)), logit_scale=1.0,
                      layers=tuple(_layer_spec(i, l) for i, l in enumerate(cfg["layers"])), norm_offset=0.0, block_style="postnorm", position="none",
                      residual_alpha=float(cfg["postln_alpha"]), depth_average=True)


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

    def norm(name):          # one number for all coordinates
        t = ckpt.get(name)
        if t is None or t.numel() != 1:
            raise AtomaError(f"norm {name} is {None if t is None else tuple(t.shape)}, a single number is needed")
        return t.float().reshape(1).expand(W)

    def gate_up(pre, n):
        return torch.cat([get(pre + "gate", (n, W)), get(pre + "up", (n, W))], 0)

    out = {"embed": get("embed", (spec.vocab, W)), "head": get("head", (spec.vocab, W)), "embed_norm": norm("embed.norm"),
           "final_norm": norm("final.norm"), "layers": []}
    for i, ls in enumerate(spec.layers):
        p, q = f"l{i}.", f"l{i}.mix."
        w = {"norm1": norm(p + "norm1"), "depth_w": get(p + "dwa", (i + 2,))}
        if ls.softmax is not None:
            a = ls.softmax
            nq, nk, nv = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
            w.update(w_q=get(q + "q", (nq, W)), b_q=get(q + "q.b", (nq,)), w_k=get(q + "k", (nk, W)), b_k=get(q + "k.b", (nk,)),
                     w_v=get(q + "v", (nv, W)), b_v=get(q + "v.b", (nv,)), head_scale=get(q + "temp", (a.heads,)), w_o=get(q + "o", (W, a.heads * a.vdim)))
        elif ls.latent is not None:
            a = ls.latent
            w.update(w_dq=get(q + "dq", (a.q_rank, W)), dq_norm=get(q + "dq.norm", (a.q_rank,)),
                     w_uq=get(q + "uq", (a.heads * (a.dim + a.rot_dim), a.q_rank)), w_dkv=get(q + "dkv", (a.kv_rank + a.rot_dim, W)),
                     dkv_norm=get(q + "dkv.norm", (a.kv_rank,)), w_uk=get(q + "uk", (a.heads * a.dim, a.kv_rank)),
                     w_uv=get(q + "uv", (a.heads * a.vdim, a.kv_rank)), w_g=get(q + "g", (a.heads * a.vdim, W)), w_o=get(q + "o", (W, a.heads * a.vdim)))
        else:
            d = ls.lru
            S, n = d.width, d.width // d.blocks
            lam = get(q + "lam", (S,)).double()
            rate = -DECAY_FACTOR * (lam.clamp_min(0.0) + torch.log1p(torch.exp(-lam.abs())))
            w.update(w_y=get(q + "y", (S, W)), b_y=get(q + "y.b", (S,)), w_x=get(q + "x", (S, W)), b_x=get(q + "x.b", (S,)),
                     tap_w=get(q + "conv", (S, d.taps)), tap_b=get(q + "conv.b", (S,)), gate_r=get(q + "ra", (d.blocks, n, n)),
                     gate_i=get(q + "ri", (d.blocks, n, n)), gate_r_b=get(q + "ra.b", (d.blocks, n)).reshape(S),
                     gate_i_b=get(q + "ri.b", (d.blocks, n)).reshape(S), rate=rate, w_o=get(q + "o", (W, S)))
        f = p + "mlp."
        if ls.mlp is not None or ls.moe is not None:
            w["norm2"] = norm(p + "norm2")
        if ls.mlp is not None:
            w["w_gate_up"], w["w_down"] = gate_up(f, ls.mlp.ff), get(f + "down", (W, ls.mlp.ff))
        if ls.moe is not None:
            e = ls.moe
            w["w_router"] = get(f + "router", (e.experts, W))
            w["router_correction"] = get(f + "correction", (e.experts,))
            w["w_expert_gate_up"] = torch.stack([gate_up(f"{f}e{k}.", e.ff) for k in range(e.experts)])
            w["w_expert_down"] = torch.stack([get(f"{f}e{k}.down", (W, e.ff)) for k in range(e.experts)])
            if e.shared_ff > 0:
                w["w_ff_in"], w["w_down"] = gate_up(f + "shared.", e.shared_ff), get(f + "shared.down", (W, e.shared_ff))
        out["layers"].append(w)
    return out
