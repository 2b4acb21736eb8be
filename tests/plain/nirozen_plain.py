"""Plain Nirozen decoder: whole sequences, no cache, one function per mechanism.

Nirozen is a pre-norm decoder without rotated positions: what tells a token its place is a sinusoidal vector added to the
embedding, beside a row of a hashed table of token pairs. Its mixer is attention through low-rank latents whose softmax
has a learned sink per head and whose output is gated channel by channel; its feed-forward is a mixture of SiLU experts
weighted by the softmax over the chosen logits, with a shared expert; its norms keep their gains around zero; a run of
layers may be applied several times, each pass entered by adding a vector of its own.

Everything runs on the CPU with ordinary tensor operations in the dtype ``work`` (float32 or float64). Nothing here is
imported by the product path and nothing of the product path is imported here. ``cfg`` is the parsed ``config.json``;
``w`` maps checkpoint names to tensors.
"""

from __future__ import annotations

import torch


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def centred_norm(x, gain, eps):
    """RMS norm whose stored gain is the distance from one."""
    return rms(x, eps) * (1.0 + gain)


def silu(z):
    return z * torch.sigmoid(z)


def pair_rows(ids, n, a, b):
    """Row of the pair table for every token of a sequence: a hash of the previous and the current token; the last row,
    number ``n``, for the first token."""
    rows = torch.full_like(ids, n)
    rows[1:] = (ids[:-1] * a + ids[1:] * b) % n
    return rows


def place_vectors(count, width, work):
    """[count, width]: column 2i holds sin(p / 10000^(2i / width)) of place p, column 2i + 1 the cosine."""
    col = torch.arange(width)
    angle = torch.arange(count, dtype=torch.float64)[:, None] * 10000.0 ** (-(2.0 * (col // 2).double()) / width)[None, :]
    return torch.where((col % 2 == 0)[None, :], torch.sin(angle), torch.cos(angle)).to(work)


def embedding(ids, w, e):
    x = w["embed"][ids] * e.get("scale", 1.0)
    bg = e.get("bigram")
    if bg:
        x = x + w["bigram"][pair_rows(ids, bg["buckets"], bg["mul_prev"], bg["mul_cur"])]
    return x + place_vectors(ids.shape[0], x.shape[-1], x.dtype)


def sink_softmax(s, sink):
    """s [heads, queries, keys] (unseen keys at -inf): exp(s) over the sum of the seen keys' exp(s) plus exp(sink of the head)."""
    top = torch.maximum(s.amax(dim=-1, keepdim=True), sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def causal_sink_attention(q, k, v, scale, sink):
    """q, k [tokens, heads, dk], v [tokens, heads, dv]: token i attends to every j <= i and to its head's sink."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    later = torch.ones(T, T, dtype=torch.bool).triu(1)
    return torch.einsum("hij,jhd->ihd", sink_softmax(s.masked_fill(later, float("-inf")), sink), v)


def latent_attention(h, w, p, m, eps):
    """The mixer. ``m``: its sizes from config.json; ``p``: tensor-name prefix ('l3.mix.')."""
    T, H = h.shape[0], m["heads"]
    c_q = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    c = rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    q = (c_q @ w[p + "uq"].T).reshape(T, H, m["dim"])
    k = (c @ w[p + "uk"].T).reshape(T, H, m["dim"])
    v = (c @ w[p + "uv"].T).reshape(T, H, m["vdim"])
    o = causal_sink_attention(q, k, v, m["scale"], w[p + "sink"]).reshape(T, H * m["vdim"])
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated_mlp(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert_choice(h, w, p, f):
    """(indices [tokens, top], weights [tokens, top], margin [tokens]): the ``top`` experts with the largest logits, the
    softmax over those logits; ``margin`` is the gap between the last chosen and the first refused logit."""
    top = f["router"]["top"]
    z = h @ w[p + "router"].T + w[p + "router.b"]
    val, idx = torch.sort(z, dim=-1, descending=True, stable=True)
    margin = val[:, top - 1] - val[:, top] if top < z.shape[-1] else torch.full_like(val[:, 0], float("inf"))
    return idx[:, :top], torch.softmax(val[:, :top], dim=-1), margin


def routed_experts(h, w, p, f, margins=None):
    idx, wt, margin = expert_choice(h, w, p, f)
    if margins is not None:
        margins.append(margin)
    out = torch.zeros(h.shape[0], w[p + "e0.down"].shape[0], dtype=h.dtype)
    for e in range(f["router"]["experts"]):
        share = (wt * (idx == e)).sum(dim=-1, keepdim=True)
        out = out + share * gated_mlp(h, w, p + f"e{e}.")
    if f.get("shared"):
        out = out + gated_mlp(h, w, p + "shared.")
    return out


def layer(x, w, i, L, eps, margins=None):
    p = f"l{i}."
    if L["type"] != "latent_attention":
        raise ValueError(f"layer {i}: unknown mixer {L['type']!r}")
    x = x + latent_attention(centred_norm(x, w[p + "norm1"], eps), w, p + "mix.", L["mixer"], eps)
    if L.get("mlp") is not None:
        x = x + routed_experts(centred_norm(x, w[p + "norm2"], eps), w, p + "mlp.", L["mlp"], margins)
    return x


def layer_runs(cfg):
    """The order in which layers are applied: [(layer index, pass number where a pass begins here, else None)]."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop or loop["stop"] <= loop["start"]:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg, w, tokens, work=torch.float64, keep_stream=False, margins=None):
    """Logits [tokens, vocab] of one sequence (and, if asked, the stream after every layer application). ``margins``: a
    list that receives, for every run of a layer with experts, by how much each token's choice of experts was clear."""
    w = {k: (v.to(work) if v.is_floating_point() else v) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = embedding(ids, w, cfg.get("embedding") or {})
    kept = []
    for i, t in layer_runs(cfg):
        if t is not None:
            x = x + w["loop.step"][t]
        x = layer(x, w, i, cfg["layers"][i], eps, margins)
        kept.append(x)
    logits = centred_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(kept)) if keep_stream else logits


def greedy_generate(cfg, w, prompt, n, work=torch.float64):
    """The ``n`` tokens that always taking the largest logit gives after ``prompt`` (the whole sequence is run again
    for every token: slow and plain)."""
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(torch.argmax(forward(cfg, w, seq, work)[-1]))
        out.append(tok)
        seq.append(tok)
    return out
