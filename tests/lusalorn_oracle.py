"""Plain float64 restatement of the Lusalorn design: one function per mechanism, Python loops, whole sequences, no paging, no
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


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def unit_rms(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


# ---- the residual stream ----
def offset_norm(v, w, eps):
    """RMS norm whose weight is stored as the distance from one."""
    return unit_rms(v, eps) * (1.0 + w)


def branch_norm(x, y, m, w, eps):
    """The sublayer's result is normed, the stream is not."""
    return x + m * offset_norm(y, w, eps)


def embedding(tokens, P, bigram=None):
    """Rows of the token table, plus a row picked by a hash of the pair (token before, token); a sequence's first token has a row of its
    own behind the hashed ones."""
    x = P["embed"][torch.as_tensor(tokens)].clone()
    if bigram is None:
        return x
    n, prev, cur = int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"])
    for t, tok in enumerate(tokens):
        row = n if t == 0 else (int(tokens[t - 1]) * prev + int(tok) * cur) % n
        x[t] += P["bigram"][row]
    return x


# ---- rotations ----
def rotary_frequencies(rot):
    """(dims / 2 frequencies, amplitude): base^(-2i / dims); `scaling` {factor, original, fast, slow} divides slow pairs by factor, keeps
    fast ones and blends linearly in the pair's index in between; cos and sin are then scaled by 0.1 ln(factor) + 1."""
    dims, base, scaling = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
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


def rotate_halves(x, positions, freqs, amplitude=1.0):
    """x [T, heads, n]: entries (i, i + len(freqs)) turned by position * freq[i] and scaled by amplitude; the rest pass unchanged."""
    out, n = x.clone(), len(freqs)
    pos = torch.as_tensor(positions, dtype=F64)
    for i in range(n):
        ang = (pos * freqs[i]).unsqueeze(-1)
        c, s = torch.cos(ang) * amplitude, torch.sin(ang) * amplitude
        u, v = x[..., i], x[..., i + n]
        out[..., i] = u * c - v * s
        out[..., i + n] = v * c + u * s
    return out


def positioned(x, rot, positions):
    if not rot or not int(rot["dims"]):
        return x
    freqs, amp = rotary_frequencies(rot)
    return rotate_halves(x, positions, freqs, amp)


# ---- attention ----
def first_visible(i, window):
    return max(0, i - window + 1) if window else 0


def window_of(m):
    return int((m.get("mask") or {}).get("size", 0))


def softmax_heads(q, k, v, key_head, value_head, scale, window):
    """q [T, H, D], k [T, *, D], v [T, *, V] -> [T, H, V]; head h reads key head key_head(h) and value head value_head(h)."""
    T, H = q.shape[:2]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        lo = first_visible(i, window)
        for h in range(H):
            out[i, h] = torch.softmax((k[lo:i + 1, key_head(h)] @ q[i, h]) * scale, 0) @ v[lo:i + 1, value_head(h)]
    return out


def grouped_attention(h, P, pre, m, eps, positions):
    """Grouped heads with weighted per-head norms of q and k before the rotation; every earlier token is visible."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ P[pre + "q"].T).reshape(T, H, D), eps) * P[pre + "q.norm"]
    k = unit_rms((h @ P[pre + "k"].T).reshape(T, G, D), eps) * P[pre + "k.norm"]
    q, k = positioned(q, m.get("rot"), positions), positioned(k, m.get("rot"), positions)
    v = (h @ P[pre + "v"].T).reshape(T, G, V)
    g = lambda hd: hd // (H // G)
    return softmax_heads(q, k, v, g, g, float(m["scale"]), 0).reshape(T, H * V) @ P[pre + "o"].T


def difference_weight(P, pre, diff):
    """The factor of the second map, one number for the layer."""
    return torch.exp((P[pre + "lq1"] * P[pre + "lk1"]).sum()) - torch.exp((P[pre + "lq2"] * P[pre + "lk2"]).sum()) + diff


def combine_maps(a1, a2, lam, diff, eps):
    """[.., V] of both maps -> their weighted difference at unit root mean square, times 1 - diff."""
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def keys_values(h, P, pre, m, eps, positions):
    T, G, D, V = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    k = unit_rms((h @ P[pre + "k"].T + P[pre + "k.b"]).reshape(T, 2 * G, D), eps) * P[pre + "k.norm"]
    return positioned(k, m.get("rot"), positions), (h @ P[pre + "v"].T + P[pre + "v.b"]).reshape(T, G, V)


def differential_attention(h, P, pre, m, eps, positions, kv):
    """Two softmax maps per head over the same values, windowed.  kv: (keys [T, 2 G, D] as group by group [map 1, map 2], values [T, G, V]),
    this layer's own or an earlier layer's."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    k, v = kv
    q = unit_rms((h @ P[pre + "q"].T + P[pre + "q.b"]).reshape(T, 2 * H, D), eps) * P[pre + "q.norm"]
    q = positioned(q, m.get("rot"), positions)
    g = lambda hd: hd // (H // G)
    scale, window = float(m["scale"]), window_of(m)
    a = [softmax_heads(q[:, n::2], k[:, n::2], v, g, g, scale, window) for n in (0, 1)]
    o = combine_maps(a[0], a[1], difference_weight(P, pre, float(m["diff"])), float(m["diff"]), eps)
    return o.reshape(T, H * V) @ P[pre + "o"].T + P[pre + "o.b"]


# ---- state-space recurrence ----
def causal_conv(x, w, bias):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x) + bias
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j] * x[:T - back]
    return out


def state_space(x, B, C, dt, A_log, D):
    """x [T, H, V], B and C [T, G, N], dt [T, H] (already positive): S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x, from zero."""
    T, H, V = x.shape
    per = H // B.shape[1]
    S, y = torch.zeros(H, B.shape[2], V, dtype=F64), torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // per
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y


def gate_then_norm(y, z, weight, parts, eps):
    """The gate comes first; every one of `parts` equal parts has its own root mean square."""
    u = y * silu(z)
    T, n = u.shape
    return unit_rms(u.reshape(T, parts, n // parts), eps).reshape(T, n) * weight


def state_space_block(h, P, pre, m, eps):
    T, H, V, G, N = h.shape[0], m["heads"], m["vdim"], m["groups"], m["state"]
    inner = H * V
    z, xbc, dt = torch.split(h @ P[pre + "in"].T, [inner, inner + 2 * G * N, H], 1)
    u = silu(causal_conv(xbc, P[pre + "conv"], P[pre + "conv.b"]))
    x, B, C = torch.split(u, [inner, G * N, G * N], 1)
    y = state_space(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + P[pre + "dt_bias"]), P[pre + "A_log"], P[pre + "D"])
    return gate_then_norm(y.reshape(T, inner), z, P[pre + "norm"], m["norm_groups"], eps) @ P[pre + "o"].T


# ---- feed-forward ----
def gated_ff(h, P, pre):
    return (silu(h @ P[pre + "gate"].T) * (h @ P[pre + "up"].T)) @ P[pre + "down"].T


# ---- the model ----
def forward(cfg, P, tokens):
    """tokens -> (logits [T, vocab], the stream after every layer [layers, T, width]), float64."""
    P = {k: v.to(F64) for k, v in P.items()}
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    positions = list(range(len(tokens)))
    x = embedding(tokens, P, (cfg.get("embedding") or {}).get("bigram"))
    trace, caches = [], {}
    for i, lc in enumerate(cfg["layers"]):
        pre, m = f"l{i}.mix.", lc["mixer"]
        if lc["type"] == "attention":
            j = m.get("kv_from")
            if j is None:
                caches[i] = keys_values(x, P, pre, m, eps, positions)
            y = differential_attention(x, P, pre, m, eps, positions, caches[i if j is None else j])
        elif lc["type"] == "parallel":
            y = (float(m["left_scale"]) * grouped_attention(x, P, pre + "left.", m["left"], eps, positions)
                 + float(m["right_scale"]) * state_space_block(x, P, pre + "right.", m["right"], eps))
        else:
            raise ValueError(lc["type"])
        x = branch_norm(x, y, mult, P[f"l{i}.norm1"], eps)
        if lc.get("mlp") is not None:
            x = branch_norm(x, gated_ff(x, P, f"l{i}.mlp."), mult, P[f"l{i}.norm2"], eps)
        trace.append(x)
    return offset_norm(x, P["final.norm"], eps) @ P["head"].T, torch.stack(trace)


# ---- random small models for the tests ----
def copied(x):
    return json.loads(json.dumps(x))


def random_config(width=56, vocab=67, kinds=("attention", "parallel", "shared"), mlps=True, ff=44, mult=0.8, eps=1e-5, attention=None, shared=None,
                  left=None, right=None, scales=(0.7, 1.3), bigram=(97, 31, 5)):
    """A configuration in the checkpoint's format.  `kinds`: "attention", "shared" (attention on the keys and values of the last
    "attention" layer before it) or "parallel"; sizes by keyword (`shared` overrides what such a layer may choose for itself); `mlps`: one
    flag or one per layer; bigram = None: no pair table."""
    a_ = dict(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, diff=0.35, mask=dict(size=21), rot=dict(base=3000.0, dims=8))
    l_ = dict(heads=4, kv_heads=2, dim=24, vdim=16, scale=0.25, rot=dict(base=5000.0, dims=16, scaling=dict(factor=6.0, original=128, fast=8.0, slow=1.0)))
    r_ = dict(heads=6, vdim=12, groups=3, state=20, norm_groups=2, conv=4)
    for base, over in ((a_, attention), (l_, left), (r_, right)):
        base.update(over or {})
    s_ = dict(copied(a_), **(shared or {}))
    layers, source = [], None
    for i, kind in enumerate(kinds):
        if kind == "parallel":
            m = dict(left=copied(l_), right=copied(r_), left_scale=scales[0], right_scale=scales[1])
        else:
            m = copied(a_ if kind == "attention" else s_)
            if kind == "attention":
                source = i
            else:
                m["kv_from"] = source
        with_ff = mlps[i] if isinstance(mlps, (list, tuple)) else mlps
        layers.append(dict(type="parallel" if kind == "parallel" else "attention", mixer=m, mlp=dict(kind="dense", ff=ff) if with_ff else None))
    cfg = dict(architecture="Lusalorn", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, layers=layers)
    if bigram:
        cfg["embedding"] = dict(bigram=dict(buckets=bigram[0], mul_prev=bigram[1], mul_cur=bigram[2]))
    return cfg


def random_weights(cfg, g):
    """float32 tensors under the checkpoint's names, already rounded to bfloat16 values (so that a bfloat16 file holds them exactly)."""
    W, P = cfg["width"], {}

    def rnd(*shape, scale=1.0, shift=0.0):
        return ((torch.randn(shape, generator=g) * scale + shift).to(torch.bfloat16)).float()

    def lin(out, inp, gain=1.0):
        return rnd(out, inp, scale=gain * inp ** -0.5)

    P["embed"], P["head"], P["final.norm"] = rnd(cfg["vocab"], W), lin(cfg["vocab"], W), rnd(W, scale=0.2)
    big = (cfg.get("embedding") or {}).get("bigram")
    if big:
        P["bigram"] = rnd(big["buckets"] + 1, W, scale=0.7)
    for i, l in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", l["mixer"], f"l{i}.mix."
        P[p + "norm1"] = rnd(W, scale=0.2)
        if l["type"] == "attention":
            H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            own = m.get("kv_from") is None
            for n, rows in (("q", 2 * H * D),) + ((("k", 2 * G * D), ("v", G * V)) if own else ()):
                P[q + n], P[q + n + ".b"] = lin(rows, W), rnd(rows, scale=0.5)
            for n in ("q",) + (("k",) if own else ()):
                P[q + n + ".norm"] = rnd(D, scale=0.2, shift=1.3)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                P[q + n] = rnd(D, scale=0.15)
            P[q + "o"], P[q + "o.b"] = lin(W, H * V), rnd(W, scale=0.3)
        else:
            a, d = m["left"], m["right"]
            H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * V)):
                P[q + "left." + n] = lin(rows, W)
            P[q + "left.q.norm"], P[q + "left.k.norm"] = rnd(D, scale=0.2, shift=1.4), rnd(D, scale=0.2, shift=1.4)
            P[q + "left.o"] = lin(W, H * V, 2.0)
            inner, chan = d["heads"] * d["vdim"], d["heads"] * d["vdim"] + 2 * d["groups"] * d["state"]
            r = q + "right."
            P[r + "in"] = lin(inner + chan + d["heads"], W)
            P[r + "conv"], P[r + "conv.b"] = rnd(chan, d["conv"], scale=0.6), rnd(chan, scale=0.3)
            P[r + "dt_bias"], P[r + "A_log"], P[r + "D"] = rnd(d["heads"], shift=-1.5), rnd(d["heads"], shift=-0.5), rnd(d["heads"])
            P[r + "norm"], P[r + "o"] = rnd(inner, scale=0.2, shift=1.0), lin(W, inner)
        if l.get("mlp") is not None:
            f, n = p + "mlp.", l["mlp"]["ff"]
            P[p + "norm2"] = rnd(W, scale=0.2)
            P[f + "gate"], P[f + "up"], P[f + "down"] = lin(n, W, 1.5), lin(n, W), lin(W, n)
    return P
