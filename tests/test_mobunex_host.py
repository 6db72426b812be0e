"""Mobunex's configuration and checkpoint reading (host only): sizes and constants from the configuration, optional parts, the names
and shapes wanted from a checkpoint, errors for what the design does not have; and the plain implementation's own arithmetic."""
import math

import pytest
import torch

import mobunex_oracle as mo
from atoma_infer_b200 import mobunex, models
from atoma_infer_b200.hybrid import RotarySpec
from atoma_infer_b200.ops import AtomaError


def test_spec_reads_every_size_and_constant_from_the_configuration():
    cfg = mo.random_config(width=56, vocab=83, kinds=("rglru", "attention", "latent_attention"), mlps=("dense", None, "moe"), ff=72, alpha=3.5, eps=3e-6,
                           attention=dict(heads=6, kv_heads=3, dim=32, vdim=8, scale=0.11, mask=dict(size=19)),
                           latent=dict(heads=5, dim=24, rot_dim=16, vdim=8, q_rank=20, kv_rank=48, scale=0.3, mask=dict(size=7),
                                       rot=dict(base=777.0, dims=16, scaling=dict(factor=5.0, original=96, fast=6.0, slow=2.0))),
                           rglru=dict(width=40, blocks=5, conv=3), router=dict(experts=12, top=4, groups=dict(count=6, keep=2)), expert_ff=26, shared_ff=18)
    spec = mobunex.spec_from_config(cfg)
    assert (spec.width, spec.vocab, spec.eps, spec.block_style, spec.norm_offset, spec.logit_scale) == (56, 83, 3e-6, "postnorm", 0.0, 1.0)
    assert (spec.residual_alpha, spec.depth_average, spec.has_state) == (3.5, True, True)
    assert [l.mixer for l in spec.layers] == ["lru", "softmax_attention", "latent_attention"]
    d = spec.layers[0].lru
    assert (d.width, d.blocks, d.taps, d.act) == (40, 5, 3, "gelu_tanh")
    assert spec.layers[0].mlp.ff == 72 and spec.layers[0].mlp.act == "silu" and spec.layers[0].moe is None
    a = spec.layers[1].softmax
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.bias, a.head_scale) == (6, 3, 32, 8, 0.11, 19, True, True)
    assert spec.layers[1].mlp is None and spec.layers[1].moe is None
    m = spec.layers[2].latent
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.window, m.out_gate) == (5, 24, 16, 8, 20, 48, 0.3, 7, True)
    assert (m.rotary.dims, m.rotary.base, m.rotary.interleaved, m.rotary.yarn) == (16, 777.0, True, (5.0, 96.0, 6.0, 2.0))
    e = spec.layers[2].moe
    assert (e.experts, e.top, e.ff, e.shared_ff, e.groups, e.keep_groups, e.group_top) == (12, 4, 26, 18, 6, 2, 2)
    assert (e.score, e.correction, e.renormalize, e.scale_input, e.identity, e.alpha, e.up_shift, e.limit) == ("sigmoid", True, True, False, 0, 1.0, 0.0, 0.0)
    assert models.resolve(cfg).name == "Mobunex" and models.resolve(cfg).needs_state(cfg)
    # cache bytes of a token: keys and values of the attention layer, latent and rotated key part of the latent layer
    assert spec.cache_bytes_per_token(torch.bfloat16) == 2 * (3 * (32 + 8) + 48 + 16)


def test_optional_parts():
    cfg = mo.random_config(kinds=("attention", "latent_attention"), mlps=("moe", "moe"), shared_ff=0, router=dict(groups=None), attention=dict(mask=None),
                           latent=dict(rot=dict(base=100.0, dims=8)))
    del cfg["layers"][1]["mixer"]["mask"]
    spec = mobunex.spec_from_config(cfg)
    assert spec.layers[0].softmax.window == 0 and spec.layers[1].latent.window == 0 and spec.layers[1].latent.rotary.yarn is None
    assert (spec.layers[0].moe.shared_ff, spec.layers[0].moe.groups) == (0, 1)
    assert not spec.has_state and not models.resolve(cfg).needs_state(cfg)
    w = mobunex.weights_from_checkpoint(spec, mo.random_weights(cfg, torch.Generator().manual_seed(0)))
    assert "w_ff_in" not in w["layers"][0] and tuple(w["layers"][0]["w_expert_down"].shape) == (8, 48, 24)


def test_checkpoint_names_and_shapes():
    cfg = mo.random_config(kinds=("rglru", "attention", "latent_attention"), mlps=("moe", "dense", None))
    P = mo.random_weights(cfg, torch.Generator().manual_seed(2))
    spec = mobunex.spec_from_config(cfg)
    out = mobunex.weights_from_checkpoint(spec, P)
    W = cfg["width"]
    assert tuple(out["embed_norm"].shape) == (W,) and float(out["embed_norm"][3]) == float(P["embed.norm"])
    l0, l1, l2 = out["layers"]
    assert tuple(l0["depth_w"].shape) == (2,) and tuple(l2["depth_w"].shape) == (4,)
    assert torch.equal(l0["w_expert_gate_up"][5], torch.cat([P["l0.mlp.e5.gate"], P["l0.mlp.e5.up"]]))
    assert torch.equal(l0["w_expert_down"][7], P["l0.mlp.e7.down"]) and torch.equal(l0["router_correction"], P["l0.mlp.correction"])
    assert torch.equal(l0["w_ff_in"], torch.cat([P["l0.mlp.shared.gate"], P["l0.mlp.shared.up"]])) and torch.equal(l0["w_down"], P["l0.mlp.shared.down"])
    n = cfg["layers"][0]["mixer"]["width"]
    assert tuple(l0["gate_r_b"].shape) == (n,) and torch.equal(l0["gate_i"], P["l0.mix.ri"])
    assert torch.allclose(l0["rate"].double(), -8.0 * torch.log1p(torch.exp(P["l0.mix.lam"].double())), rtol=1e-12)
    assert torch.equal(l1["head_scale"], P["l1.mix.temp"]) and torch.equal(l1["b_v"], P["l1.mix.v.b"])
    assert torch.equal(l1["w_gate_up"], torch.cat([P["l1.mlp.gate"], P["l1.mlp.up"]]))
    assert torch.equal(l2["w_g"], P["l2.mix.g"]) and "norm2" not in l2
    for name, bad in (("l0.mix.lam", None), ("l2.dwa", torch.zeros(3)), ("l1.mix.q.b", None), ("l0.norm1", torch.zeros(W)), ("final.norm", None)):
        broken = dict(P)
        if bad is None:
            del broken[name]
        else:
            broken[name] = bad
        with pytest.raises(AtomaError, match=name):
            mobunex.weights_from_checkpoint(spec, broken)


def test_what_the_design_does_not_have_is_refused():
    cfg = mo.random_config()
    for path, value, words in ((("layers", 0, "type"), "gla", "gla"), (("layers", 1, "mlp", "kind"), "switch", "switch"),
                               (("layers", 0, "mixer", "mask"), dict(size=0), "window")):
        other = mo.copied(cfg)
        at = other
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(AtomaError, match=words):
            mobunex.spec_from_config(other)


@pytest.mark.parametrize("dims,base,scaling", [(24, 30000.0, (6.0, 2048, 24.0, 1.5)), (16, 100.0, (4.0, 64, 4.0, 0.5)), (8, 1e6, (2.0, 8, 1.0, 1.0))])
def test_yarn_rule(dims, base, scaling):
    """Fast pairs keep their frequency, slow pairs have it divided, the share in between grows with the index."""
    r = RotarySpec(dims=dims, base=base, interleaved=True, yarn=scaling)
    plain = RotarySpec(dims=dims, base=base).frequencies()
    f, amp = mo.yarn_frequencies(dims, base, dict(zip(("factor", "original", "fast", "slow"), scaling)))
    got = r.frequencies()
    assert all(abs(a - float(b)) < 1e-15 for a, b in zip(got, f)) and r.amplitude == amp == 0.1 * math.log(scaling[0]) + 1.0
    share = [(p - q) / (p - p / scaling[0]) for p, q in zip(plain, got)]
    assert all(-1e-12 < s < 1 + 1e-12 for s in share) and all(b >= a - 1e-12 for a, b in zip(share, share[1:]))


def test_plain_window_and_recurrence():
    """The plain implementation itself: who is visible, and a recurrence whose closed form is known."""
    assert [mo.first_visible(i, 3) for i in range(6)] == [0, 0, 0, 1, 2, 3] and mo.first_visible(9, 0) == 0
    u, r, i = torch.ones(5, 1, dtype=mo.F64), torch.ones(5, 1, dtype=mo.F64), torch.ones(5, 1, dtype=mo.F64)
    lam = torch.tensor([math.log(math.expm1(math.log(2.0) / 8.0))], dtype=mo.F64)      # log a = -ln 2
    S = mo.gated_linear_recurrence(u, r, i, lam)[:, 0]
    b = math.sqrt(0.75)
    assert torch.allclose(S, torch.tensor([b * (2 - 0.5 ** t) for t in range(5)], dtype=mo.F64), rtol=1e-12)
    assert torch.equal(mo.depth_average([torch.ones(2), torch.full((2,), 3.0)], [0.5, 2.0]), torch.full((2,), 6.5))
