"""Plain Levolix decoder: whole sequences, no cache, one function per mechanism.

Levolix normalises what a sublayer returns and nothing else: x <- x + N1(mixer(x)), then x <- x + N2(experts(x)), N an RMS
norm whose gain is stored less one; the sublayers read the stream as it is. Its mixers are a retention (linear attention
with one fixed decay a head) and a pair of mixers on the same input: an attention inside fixed chunks of positions, with
one RMS norm over the whole query and the whole key projection, neighbouring channels rotated, a one in the softmax
denominator and a sigmoid gate per channel, beside a gated delta rule (a matrix state per head from which the part that
the current key reads is taken back before the new value is written). Its feed-forward is a mixture of experts, some of
which return their input. The output matrix is the embedding table.

Everything runs on the CPU with ordinary tensor operations in the dtype ``work`` (float32 or float64). Nothing here is
imported by the product path and nothing of the product path is imported here. ``cfg`` is the parsed ``config.json``;
``w`` maps checkpoint names to tensors.
"""

from __future__ import annotations

import torch

from .qwen3_plain import read_model  # noqa: F401  (tests read model folders through this module)

UNIT_EPS = 1e-6         # inside the root of the unit vectors of the delta rule's keys and queries


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + UNIT_EPS)


def norm_about_one(x, w, eps):
    """RMS norm whose gain is stored around zero."""
    return rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def angles(positions, dims, base, work):
    """One angle per position and pair: p * base^(-2i/dims), worked out in 64-bit."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    return (positions.to(torch.float64)[:, None] * base ** (-2.0 * i / dims)[None, :]).to(work)


def rotate_halves(v, ang):
    """v [tokens, heads, n]: channel i of the first 2 * pairs turns with channel i + pairs."""
    half = ang.shape[1]
    cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]
    a, b = v[..., :half], v[..., half:2 * half]
    return torch.cat([a * cos - b * sin, b * cos + a * sin, v[..., 2 * half:]], dim=-1)


def rotate_neighbours(v, ang):
    """v [tokens, heads, n]: channel 2i of the first 2 * pairs turns with channel 2i + 1."""
    half = ang.shape[1]
    cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]
    a, b = v[..., 0:2 * half:2], v[..., 1:2 * half:2]
    turned = torch.stack([a * cos - b * sin, b * cos + a * sin], dim=-1).flatten(-2)
    return torch.cat([turned, v[..., 2 * half:]], dim=-1)


def same_chunk(T, size):
    """[T, T]: position i sees j <= i of its own chunk of ``size`` positions, counted from position 0."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))


def softmax_plus_one(s, seen):
    """exp(s_j) / (1 + sum exp(s_j)) over the seen keys."""
    s = s.masked_fill(~seen, float("-inf"))
    m = torch.clamp(s.amax(dim=-1, keepdim=True), min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


def attend(q, k, v, scale, seen):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key/value head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    kk, vv = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    p = softmax_plus_one(torch.einsum("ihd,jhd->hij", q, kk) * scale, seen)
    return torch.einsum("hij,jhd->ihd", p, vv)


def chunked_attention(h, w, p, m, eps):
    """The left mixer of 'parallel'."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + n].T + w[p + n + ".b"] for n in ("q", "k", "v"))
    q = (rms(q, eps) * w[p + "q.norm"]).reshape(T, H, d)
    k = (rms(k, eps) * w[p + "k.norm"]).reshape(T, G, d)
    ang = angles(torch.arange(T), m["rot"]["dims"], m["rot"]["base"], h.dtype)
    o = attend(rotate_neighbours(q, ang), rotate_neighbours(k, ang), v.reshape(T, G, dv), m["scale"], same_chunk(T, m["mask"]["size"]))
    o = o.reshape(T, H * dv) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def short_convolution(u, taps_w):
    """u [tokens, channels], taps_w [channels, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, C = u.shape
    taps = taps_w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + padded[j:j + T] * taps_w[:, j]
    return y


def delta_recurrence(g, beta, k, v, q, S=None):
    """g, beta [T, H], k, q [T, H, N], v [T, H, P], token by token from S (zeros when None): S <- g S, then
    u = beta (v - S^T k), S <- S + k u^T, o = S^T q. Returns (o [T, H, P], the last S [H, N, P])."""
    T, H, N = k.shape
    S = torch.zeros(H, N, v.shape[2], dtype=k.dtype) if S is None else S.clone()
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hnp,hn->hp", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, q[t]))
    return torch.stack(out), S


def head_norm_and_gate(o, gain, gate, eps):
    """o [T, H, P]: every head divided by its root mean square, times ``gain`` [P] (or None), heads side by side times
    silu(gate) [T, H * P]."""
    o = rms(o, eps)
    if gain is not None:
        o = o * gain
    return o.reshape(o.shape[0], -1) * silu(gate)


def gated_delta(h, w, p, m, eps):
    """The right mixer of 'parallel'."""
    T = h.shape[0]
    H, G, N, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, G, N)).repeat_interleave(H // G, dim=1) * N ** -0.5
    k = unit(k.reshape(T, G, N)).repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o, _ = delta_recurrence(g, beta, k, v.reshape(T, H, P), q)
    return head_norm_and_gate(o, w[p + "norm"], h @ w[p + "g"].T, eps) @ w[p + "o"].T


def decayed_recurrence(decay, k, v, q, S=None):
    """decay [H], k, q [T, H, N], v [T, H, P]: S_t = decay S_(t-1) + k_t v_t^T from S (zeros when None), o_t = S_t^T q_t.
    Returns (o [T, H, P], the last S [H, N, P])."""
    T, H, N = k.shape
    S = torch.zeros(H, N, v.shape[2], dtype=k.dtype) if S is None else S.clone()
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, q[t]))
    return torch.stack(out), S


def retention(h, w, p, m, eps):
    T = h.shape[0]
    H, N, P = m["heads"], m["dim"], m["vdim"]
    ang = angles(torch.arange(T), m["rot"]["dims"], m["rot"]["base"], h.dtype)
    q = rotate_halves((h @ w[p + "q"].T).reshape(T, H, N), ang)
    k = rotate_halves((h @ w[p + "k"].T).reshape(T, H, N), ang) * N ** -0.5
    o, _ = decayed_recurrence(torch.tensor(m["decay"], dtype=h.dtype), k, (h @ w[p + "v"].T).reshape(T, H, P), q)
    return head_norm_and_gate(o, None, h @ w[p + "g"].T, eps) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return (m["left_scale"] * chunked_attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * gated_delta(h, w, p + "right.", m["right"], eps))


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, top):
    """(scores [T, all experts], chosen [T, top]): softmax over all experts, those that return their input included; the
    correction moves the choice and never the scores."""
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    return s, torch.topk(s + w[p + "correction"], top, dim=-1).indices


def experts(h, w, p, m, margins=None):
    """``margins`` collects, per token, by how much the last chosen choice score leads the first one left out."""
    real, same, top = m["router"]["experts"], m["router"].get("identity", 0), m["router"]["top"]
    s, chosen = route(h, w, p, top)
    if margins is not None:
        c = torch.sort(s + w[p + "correction"], dim=-1, descending=True).values
        margins.append((c[:, top - 1] - c[:, top]) if top < real + same else torch.ones(h.shape[0], dtype=h.dtype))
    out = torch.zeros_like(h)
    for e in range(real + same):
        rows = (chosen == e).any(dim=-1).nonzero()[:, 0]
        if len(rows):
            y = expert(h[rows], w, f"{p}e{e}.") if e < real else h[rows]
            out[rows] += s[rows, e][:, None] * y
    return out


def forward(cfg, w, ids, work=torch.float64, margins=None):
    """(logits [T, vocab], the stream after every layer [layers, T, width]) of one sequence."""
    w = {k: (v.to(work) if v.is_floating_point() else v) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][ids]
    after = []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = {"parallel": parallel, "retention": retention}[L["type"]]
        x = x + norm_about_one(mix(x, w, p + "mix.", L["mixer"], eps), w[p + "norm1"], eps)
        if L.get("mlp") is not None:
            x = x + norm_about_one(experts(x, w, p + "mlp.", L["mlp"], margins), w[p + "norm2"], eps)
        after.append(x)
    return norm_about_one(x, w["final.norm"], eps) @ w["embed"].T, torch.stack(after)


def greedy_generate(cfg, w, prompt, n, work=torch.float64):
    """The ``n`` tokens that always taking the largest logit gives after ``prompt`` (the whole sequence is run again for
    every token: slow and plain)."""
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(torch.argmax(forward(cfg, w, torch.tensor(seq), work)[0][-1]))
        out.append(tok)
        seq.append(tok)
    return out
