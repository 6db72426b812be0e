"""Plain float64 restatement of the Mobunex design: one function per mechanism, Python loops, whole sequences, no paging, no
batching, no carried state.  It shares no code with the package; the GPU tests compare the framework against it.

Notation: matrices are stored [out, in] and applied as `h @ W.T`; sigma is the logistic function; P are the weights by their
checkpoint names.
"""
import json
import math

import torch

F64 = torch.float64


def sigma(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigma(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def unit_rms(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


# ---- the residual stream ----
def scalar_norm(v, g, eps):
    """RMS norm whose weight is ONE number for all coordinates."""
    return unit_rms(v, eps) * g


def post_norm(x, y, alpha, g, eps):
    """The norm follows the sum: the stream times alpha plus the sublayer's result."""
    return scalar_norm(alpha * x + y, g, eps)


def depth_average(rows, weights):
    """rows: the embedding output and every layer's result so far; the next layer reads their weighted sum."""
    out = torch.zeros_like(rows[-1])
    for w, r in zip(weights, rows):
        out = out + w * r
    return out


# ---- rotations ----
def yarn_frequencies(dims, base, scaling=None):
    """(dims / 2 frequencies, amplitude): base^(-2i / dims); `scaling` {factor, original, fast, slow} divides slow pairs by factor, keeps
    fast ones and blends linearly in the pair's index in between; cos and sin are then scaled by 0.1 ln(factor) + 1."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=F64), 1.0
    factor, original, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))

    def index_of(turns):      # the (real) pair index whose wavelength fits `turns` times into the original length
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(index_of(fast)), 0), min(math.ceil(index_of(slow)), dims - 1)
    out = []
    for i in range(dims // 2):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i] / factor * r + f[i] * (1.0 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, positions, freqs, amplitude=1.0):
    """x [T, ..., n]: entries (2i, 2i + 1), i < len(freqs), turned by position * freq[i] and scaled by amplitude; the rest pass unchanged."""
    out = x.clone()
    for i, f in enumerate(freqs.tolist()):
        ang = torch.as_tensor(positions, dtype=F64) * f
        while ang.dim() < x.dim() - 1:
            ang = ang.unsqueeze(-1)
        c, s = torch.cos(ang) * amplitude, torch.sin(ang) * amplitude
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ---- mixers ----
def first_visible(i, window):
    return max(0, i - window + 1) if window else 0


def window_of(m):
    return int((m.get("mask") or {}).get("size", 0))


def windowed_softmax(scores_of, values_of, T, H, V, window):
    """out[i, h] = softmax over the visible keys j of scores_of(i, h, lo, hi) times values_of(h, lo, hi)."""
    out = torch.zeros(T, H, V, dtype=F64)
    for i in range(T):
        lo = first_visible(i, window)
        for h in range(H):
            out[i, h] = torch.softmax(scores_of(i, h, lo, i + 1), 0) @ values_of(h, lo, i + 1)
    return out


def grouped_attention(h, P, pre, m, eps):
    """Grouped heads with projection biases, unweighted per-head norms of q and k, and a factor of its own per head on the score."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ P[pre + "q"].T + P[pre + "q.b"]).reshape(T, H, D), eps)
    k = unit_rms((h @ P[pre + "k"].T + P[pre + "k.b"]).reshape(T, G, D), eps)
    v = (h @ P[pre + "v"].T + P[pre + "v.b"]).reshape(T, G, V)
    temp, scale = P[pre + "temp"], float(m["scale"])
    g = lambda hd: hd // (H // G)
    out = windowed_softmax(lambda i, hd, lo, hi: (k[lo:hi, g(hd)] @ q[i, hd]) * scale * temp[hd], lambda hd, lo, hi: v[lo:hi, g(hd)], T, H, V, window_of(m))
    return out.reshape(T, H * V) @ P[pre + "o"].T


def latent_attention(h, P, pre, m, eps, positions):
    """Queries through a normed latent, keys and values from a normed shared latent, one rotated key part for all heads, a sigmoid gate on
    the heads' outputs."""
    T = h.shape[0]
    H, D, Rd, V, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m["rot"]
    freqs, amp = yarn_frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
    c_q = unit_rms(h @ P[pre + "dq"].T, eps) * P[pre + "dq.norm"]
    q = (c_q @ P[pre + "uq"].T).reshape(T, H, D + Rd)
    q_plain, q_rot = q[..., :D], rotate_pairs(q[..., D:], positions, freqs, amp)
    dkv = h @ P[pre + "dkv"].T
    c = unit_rms(dkv[:, :R], eps) * P[pre + "dkv.norm"]
    k_rot = rotate_pairs(dkv[:, R:], positions, freqs, amp)
    k_plain, v = (c @ P[pre + "uk"].T).reshape(T, H, D), (c @ P[pre + "uv"].T).reshape(T, H, V)
    scale = float(m["scale"])
    out = windowed_softmax(lambda i, hd, lo, hi: (k_plain[lo:hi, hd] @ q_plain[i, hd] + k_rot[lo:hi] @ q_rot[i, hd]) * scale,
                           lambda hd, lo, hi: v[lo:hi, hd], T, H, V, window_of(m))
    return (out.reshape(T, H * V) * sigma(h @ P[pre + "g"].T)) @ P[pre + "o"].T


def causal_conv(x, w, bias):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x) + bias
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j] * x[:T - back]
    return out


def blockwise(u, w, b):
    """u [T, C] in w.shape[0] equal parts, each through its own square matrix [out, in] and bias."""
    n, s = w.shape[0], w.shape[1]
    return torch.cat([u[:, i * s:(i + 1) * s] @ w[i].T + b[i] for i in range(n)], 1)


def gated_linear_recurrence(u, r, i, lam):
    """S <- a S + sqrt(1 - a^2) i u with log a = -8 r softplus(lam), from zero; every S."""
    log_a = -8.0 * r * softplus(lam)
    a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a))
    S, out = torch.zeros(u.shape[1], dtype=F64), torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + b[t] * i[t] * u[t]
        out[t] = S
    return out


def recurrent_block(h, P, pre, m):
    y = gelu_tanh(h @ P[pre + "y"].T + P[pre + "y.b"])
    u = causal_conv(h @ P[pre + "x"].T + P[pre + "x.b"], P[pre + "conv"], P[pre + "conv.b"])
    r, i = sigma(blockwise(u, P[pre + "ra"], P[pre + "ra.b"])), sigma(blockwise(u, P[pre + "ri"], P[pre + "ri.b"]))
    return (gated_linear_recurrence(u, r, i, P[pre + "lam"]) * y) @ P[pre + "o"].T


# ---- feed-forward ----
def gated_ff(h, P, pre):
    return (silu(h @ P[pre + "gate"].T) * (h @ P[pre + "up"].T)) @ P[pre + "down"].T


def route(h_row, P, pre, router):
    """One token: [(expert, weight)].  A group's score is the sum of its two largest choice scores; outside the best groups nothing can be
    chosen; ties go to the lower index."""
    s = sigma(P[pre + "router"] @ h_row)
    c = s + P[pre + "correction"] if pre + "correction" in P else s.clone()
    n, groups = router["experts"], router.get("groups")
    allowed = list(range(n))
    if groups:
        per = n // groups["count"]
        score = [sum(sorted(c[g * per:(g + 1) * per].tolist(), reverse=True)[:2]) for g in range(groups["count"])]
        best = sorted(range(groups["count"]), key=lambda g: (-score[g], g))[:groups["keep"]]
        allowed = [e for e in allowed if e // per in best]
    chosen = sorted(allowed, key=lambda e: (-float(c[e]), e))[:router["top"]]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    return [(e, float(s[e]) / total) for e in chosen]


def moe_ff(h, P, pre, mlp):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in route(h[t], P, pre, mlp["router"]):
            out[t] += w * gated_ff(h[t:t + 1], P, f"{pre}e{e}.")[0]
    return out + gated_ff(h, P, pre + "shared.") if mlp.get("shared") else out


def feed_forward(h, P, pre, mlp):
    return moe_ff(h, P, pre, mlp) if mlp["kind"] == "moe" else gated_ff(h, P, pre)


# ---- the model ----
def mixer(x, P, i, lc, eps, positions):
    pre = f"l{i}.mix."
    if lc["type"] == "attention":
        return grouped_attention(x, P, pre, lc["mixer"], eps)
    if lc["type"] == "latent_attention":
        return latent_attention(x, P, pre, lc["mixer"], eps, positions)
    if lc["type"] == "rglru":
        return recurrent_block(x, P, pre, lc["mixer"])
    raise ValueError(lc["type"])


def forward(cfg, P, tokens):
    """tokens -> (logits [T, vocab], what every layer hands on [layers, T, width]), float64."""
    P = {k: v.to(F64) for k, v in P.items()}
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    positions = list(range(len(tokens)))
    x = scalar_norm(P["embed"][torch.as_tensor(tokens)], P["embed.norm"], eps)
    rows, trace = [x], []
    for i, lc in enumerate(cfg["layers"]):
        x = post_norm(x, mixer(x, P, i, lc, eps, positions), alpha, P[f"l{i}.norm1"], eps)
        if lc.get("mlp") is not None:
            x = post_norm(x, feed_forward(x, P, f"l{i}.mlp.", lc["mlp"]), alpha, P[f"l{i}.norm2"], eps)
        rows.append(x)
        x = depth_average(rows, P[f"l{i}.dwa"])
        trace.append(x)
    return scalar_norm(x, P["final.norm"], eps) @ P["head"].T, torch.stack(trace)


# ---- random small models for the tests ----
def copied(x):
    return json.loads(json.dumps(x))


def random_config(width=48, vocab=61, kinds=("attention", "rglru", "latent_attention"), mlps=("dense", "moe", "moe"), ff=40, alpha=2.5, eps=1e-5,
                  attention=None, latent=None, rglru=None, router=None, expert_ff=24, shared_ff=16):
    """A configuration in the checkpoint's format.  `mlps`: per layer "dense", "moe" or None; sizes by keyword; shared_ff = 0: no shared expert."""
    a_ = dict(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.25, mask=dict(size=21))
    l_ = dict(heads=3, dim=16, rot_dim=8, vdim=16, q_rank=24, kv_rank=32, scale=0.2, mask=dict(size=33),
              rot=dict(base=5000.0, dims=8, scaling=dict(factor=6.0, original=128, fast=8.0, slow=1.0)))
    r_ = dict(width=60, blocks=3, conv=4)
    e_ = dict(experts=8, top=3, groups=dict(count=4, keep=2))
    for base, over in ((a_, attention), (l_, latent), (r_, rglru), (e_, router)):
        base.update(over or {})
    layers = []
    for kind, mlp in zip(kinds, mlps):
        f = None
        if mlp == "dense":
            f = dict(kind="dense", ff=ff)
        elif mlp == "moe":
            f = dict(kind="moe", router=copied(e_), expert=dict(ff=expert_ff))
            if f["router"].get("groups") is None:
                f["router"].pop("groups", None)
            if shared_ff:
                f["shared"] = dict(ff=shared_ff)
        layers.append(dict(type=kind, mixer=copied({"attention": a_, "latent_attention": l_, "rglru": r_}[kind]), mlp=f))
    return dict(architecture="Mobunex", vocab=vocab, width=width, norm=dict(eps=eps), postln_alpha=alpha, layers=layers)


def random_weights(cfg, g):
    """float32 tensors under the checkpoint's names, already rounded to bfloat16 values (so that a bfloat16 file holds them exactly)."""
    W, P = cfg["width"], {}

    def rnd(*shape, scale=1.0, shift=0.0):
        return ((torch.randn(shape, generator=g) * scale + shift).to(torch.bfloat16)).float()

    def lin(out, inp, gain=1.0):
        return rnd(out, inp, scale=gain * inp ** -0.5)

    P["embed"], P["embed.norm"] = rnd(cfg["vocab"], W), rnd(scale=0.2, shift=1.2)
    P["head"], P["final.norm"] = lin(cfg["vocab"], W), rnd(scale=0.2, shift=0.9)
    for i, l in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", l["mixer"], f"l{i}.mix."
        P[p + "norm1"], P[p + "dwa"] = rnd(scale=0.2, shift=1.0), rnd(i + 2, scale=0.3)
        P[p + "dwa"][-1] += 1.0
        P[p + "dwa"] = P[p + "dwa"].to(torch.bfloat16).float()
        if l["type"] == "attention":
            H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * V)):
                P[q + n], P[q + n + ".b"] = lin(rows, W), rnd(rows, scale=0.5)
            P[q + "temp"], P[q + "o"] = rnd(H, scale=0.4, shift=1.5), lin(W, H * V, 2.0)
        elif l["type"] == "latent_attention":
            H, D, Rd, V, Rq, Rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            P[q + "dq"], P[q + "dq.norm"], P[q + "uq"] = lin(Rq, W), rnd(Rq, scale=0.1, shift=1.0), lin(H * (D + Rd), Rq, 2.0)
            P[q + "dkv"], P[q + "dkv.norm"] = lin(Rk + Rd, W, 2.0), rnd(Rk, scale=0.1, shift=1.0)
            P[q + "uk"], P[q + "uv"] = lin(H * D, Rk, 2.0), lin(H * V, Rk)
            P[q + "g"], P[q + "o"] = lin(H * V, W, 2.0), lin(W, H * V, 3.0)
        else:
            S, B, K = m["width"], m["blocks"], m["conv"]
            for n in ("y", "x"):
                P[q + n], P[q + n + ".b"] = lin(S, W), rnd(S, scale=0.5)
            P[q + "conv"], P[q + "conv.b"] = rnd(S, K, scale=0.6), rnd(S, scale=0.3)
            for n in ("ra", "ri"):
                P[q + n], P[q + n + ".b"] = rnd(B, S // B, S // B, scale=(S // B) ** -0.5), rnd(B, S // B, scale=0.5)
            P[q + "lam"], P[q + "o"] = rnd(S, scale=1.5, shift=-3.0), lin(W, S, 2.0)
        f = l.get("mlp")
        if f is None:
            continue
        P[p + "norm2"] = rnd(scale=0.2, shift=1.1)

        def ff_tensors(pre, n):
            P[pre + "gate"], P[pre + "up"], P[pre + "down"] = lin(n, W, 1.5), lin(n, W), lin(W, n)

        if f["kind"] == "dense":
            ff_tensors(p + "mlp.", f["ff"])
        else:
            n = f["router"]["experts"]
            P[p + "mlp.router"], P[p + "mlp.correction"] = lin(n, W, 2.0), rnd(n, scale=0.3, shift=-0.4)
            for e in range(n):
                ff_tensors(f"{p}mlp.e{e}.", f["expert"]["ff"])
            if f.get("shared"):
                ff_tensors(p + "mlp.shared.", f["shared"]["ff"])
    return P
