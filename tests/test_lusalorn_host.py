"""Lusalorn's configuration and checkpoint reading (host only): sizes and constants from the configuration, optional parts, the names and
shapes wanted from a checkpoint, errors for what the design does not have; and the plain implementation's own arithmetic."""
import math

import pytest
import torch

import lusalorn_oracle as lo
from atoma_infer_b200 import lusalorn, models
from atoma_infer_b200.hybrid import RotarySpec
from atoma_infer_b200.ops import AtomaError


def test_spec_reads_every_size_and_constant_from_the_configuration():
    cfg = lo.random_config(width=72, vocab=83, kinds=("attention", "parallel", "shared"), mlps=(True, False, True), ff=52, mult=0.45, eps=3e-6,
                           attention=dict(heads=6, kv_heads=3, dim=32, vdim=40, scale=0.11, diff=0.55, mask=dict(size=19), rot=dict(base=123.0, dims=10)),
                           shared=dict(heads=9, scale=0.2, diff=0.15, mask=dict(size=4)),
                           left=dict(heads=8, kv_heads=4, dim=12, vdim=20, scale=0.35, rot=dict(base=777.0, dims=8, scaling=dict(factor=5.0, original=96, fast=6.0, slow=2.0))),
                           right=dict(heads=10, vdim=6, groups=5, state=14, norm_groups=4, conv=3), scales=(0.3, 1.9), bigram=(211, 12, 34))
    spec = lusalorn.spec_from_config(cfg)
    assert (spec.width, spec.vocab, spec.eps, spec.block_style, spec.norm_offset, spec.logit_scale) == (72, 83, 3e-6, "postnorm", 1.0, 1.0)
    assert (spec.branch_scale, spec.embed_norm, spec.depth_average, spec.residual_alpha, spec.has_state) == (0.45, False, False, 1.0, True)
    assert (spec.pair_table.buckets, spec.pair_table.mul_prev, spec.pair_table.mul_cur) == (211, 12, 34)
    assert [l.mixer for l in spec.layers] == ["softmax_attention", "attention_ssm", "softmax_attention"]
    a = spec.layers[0].softmax
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.maps, a.diff, a.kv_from) == (6, 3, 32, 40, 0.11, 19, 2, 0.55, None)
    assert (a.bias, a.out_bias, a.qk_norm) == (True, True, True)
    assert (a.rotary.dims, a.rotary.base, a.rotary.interleaved, a.rotary.yarn) == (10, 123.0, False, None)
    s = spec.layers[2].softmax
    assert (s.heads, s.kv_heads, s.scale, s.window, s.diff, s.kv_from) == (9, 3, 0.2, 4, 0.15, 0)
    m = spec.layers[1].mixer_sum
    assert (m.left_scale, m.right_scale) == (0.3, 1.9)
    assert (m.left.heads, m.left.kv_heads, m.left.dim, m.left.vdim, m.left.scale, m.left.window, m.left.maps, m.left.bias) == (8, 4, 12, 20, 0.35, 0, 1, False)
    assert (m.left.rotary.dims, m.left.rotary.yarn) == (8, (5.0, 96.0, 6.0, 2.0))
    assert (m.right.heads, m.right.vdim, m.right.groups, m.right.state, m.right.norm_groups, m.right.taps) == (10, 6, 5, 14, 4, 3)
    assert spec.layers[0].mlp.ff == 52 and spec.layers[1].mlp is None
    assert models.resolve(cfg).name == "Lusalorn" and models.resolve(cfg).needs_state(cfg)
    # cache bytes of a token: both maps' keys and the values of the first layer, the summed layer's; nothing for the layer on shared caches
    assert spec.cache_bytes_per_token(torch.bfloat16) == 2 * (3 * (2 * 32 + 40) + 4 * (12 + 20))


def test_optional_parts():
    cfg = lo.random_config(kinds=("attention", "shared"), mlps=False, bigram=None, attention=dict(mask=None, rot=None))
    spec = lusalorn.spec_from_config(cfg)
    assert spec.pair_table is None and not spec.has_state and not models.resolve(cfg).needs_state(cfg)
    assert spec.layers[0].softmax.window == 0 and spec.layers[0].softmax.rotary is None and spec.layers[1].softmax.kv_from == 0
    w = lusalorn.weights_from_checkpoint(spec, lo.random_weights(cfg, torch.Generator().manual_seed(0)))
    assert "pair_table" not in w and "w_k" not in w["layers"][1] and "norm2" not in w["layers"][0]


def test_checkpoint_names_and_shapes():
    cfg = lo.random_config(kinds=("attention", "parallel"))
    P = lo.random_weights(cfg, torch.Generator().manual_seed(2))
    spec = lusalorn.spec_from_config(cfg)
    out = lusalorn.weights_from_checkpoint(spec, P)
    l0, l1 = out["layers"]
    a, d = spec.layers[0].softmax, spec.layers[1].mixer_sum.right
    Q = {k: v.double() for k, v in P.items()}
    assert abs(l0["diff_lambda"] - float(lo.difference_weight(Q, "l0.mix.", a.diff))) < 1e-12
    assert tuple(l0["w_q"].shape) == (2 * a.heads * a.dim, cfg["width"])
    rows = P["l1.mix.right.in"]
    assert torch.equal(l1["r_w_z"], rows[:d.inner]) and torch.equal(l1["r_w_x"], rows[d.inner:2 * d.inner]) and torch.equal(l1["r_w_dt"], rows[-d.heads:])
    assert l1["r_w_bc"].shape[0] == 2 * d.groups * d.state
    for name in list(P):
        missing = dict(P)
        del missing[name]
        with pytest.raises(AtomaError):
            lusalorn.weights_from_checkpoint(spec, missing)
        wrong = dict(P)
        wrong[name] = torch.zeros(tuple(n + 1 for n in P[name].shape))
        with pytest.raises(AtomaError):
            lusalorn.weights_from_checkpoint(spec, wrong)


def test_what_the_design_does_not_have_is_refused():
    for change in (lambda c: c["layers"][0].update(type="rglru"), lambda c: c["layers"][0].update(mlp=dict(kind="moe", ff=4)),
                   lambda c: c["layers"][0]["mixer"].update(mask=dict(size=0))):
        cfg = lo.random_config(kinds=("attention",))
        change(cfg)
        with pytest.raises(AtomaError):
            lusalorn.spec_from_config(cfg)


def test_yarn_frequencies_follow_the_rule():
    for dims, base, sc in ((24, 30000.0, dict(factor=6.0, original=2048, fast=24.0, slow=1.5)), (44, 2e5, dict(factor=3.0, original=512, fast=32.0, slow=1.0)), (12, 500.0, None)):
        f, amp = lo.rotary_frequencies(dict(dims=dims, base=base, scaling=sc))
        r = RotarySpec(dims=dims, base=base, yarn=None if sc is None else tuple(sc[k] for k in ("factor", "original", "fast", "slow")))
        assert abs(r.amplitude - amp) < 1e-15
        assert max(abs(a - b) / b for a, b in zip(r.frequencies(), f.tolist())) < 1e-14


def test_the_plain_implementation_on_cases_with_known_answers():
    # one token: a softmax over one key returns its value
    q, k, v = torch.randn(1, 2, 4).double(), torch.randn(1, 1, 4).double(), torch.randn(1, 1, 3).double()
    assert torch.allclose(lo.softmax_heads(q, k, v, lambda h: 0, lambda h: 0, 0.5, 0), v.expand(1, 2, 3))
    # equal maps at lambda = 0: the first map at unit root mean square
    a = torch.randn(2, 3, 5).double()
    assert torch.allclose(lo.combine_maps(a, a, 0.0, 0.25, 0.0), 0.75 * lo.unit_rms(a, 0.0))
    # a constant decay g and step d: the state is a geometric sum
    T, d = 4, 0.5
    x, B, C = torch.ones(T, 1, 1).double(), torch.ones(T, 1, 1).double(), torch.ones(T, 1, 1).double()
    y = lo.state_space(x, B, C, torch.full((T, 1), d).double(), torch.zeros(1).double(), torch.tensor([2.0]).double())
    g = math.exp(-d)
    assert all(abs(float(y[t, 0, 0]) - (d * (1 - g ** (t + 1)) / (1 - g) + 2.0)) < 1e-12 for t in range(T))
    # a turn by position * 1: the quarter turn exchanges the pair
    r = lo.rotate_halves(torch.tensor([[[1.0, 0.0, 7.0]]]).double(), [math.pi / 2], torch.ones(1).double())
    assert torch.allclose(r, torch.tensor([[[0.0, 1.0, 7.0]]]).double(), atol=1e-12)
