"""Each mechanism of Nirozen alone, its kernel against the plain implementation's function: the position vector (alone and in
the pass that forms token row and pair row), gains stored less one, attention without positions over the latent cache with a
sink per head (every kernel form, slices, single tokens, loud keys far back and at page borders), whole prompts with per-head
keys and values on both prompt kernels, the output gate in the product's epilogue, the router whose logits come from a
product."""

from __future__ import annotations

import numpy as np
import pytest
import torch

from plain import nirozen_plain as plain

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
DT = {"fp32": torch.float32, "bf16": torch.bfloat16}
TOL = {"fp32": dict(rtol=2e-5, atol=2e-5), "bf16": dict(rtol=2e-2, atol=2e-2)}


def ops():
    from sleuth_b200.kernels import ops as o
    return o


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# ---- position vectors ----
def place_vectors_at(positions, width):
    """The plain position vectors of chosen positions, which may be far from 0."""
    col = torch.arange(width)
    freq = 10000.0 ** (-(2.0 * (col // 2).double()) / width)
    a = torch.tensor(positions, dtype=torch.float64)[:, None] * freq[None, :]
    return torch.where((col % 2 == 0)[None, :], torch.sin(a), torch.cos(a))


@pytest.mark.parametrize("width", [1, 2, 75, 128, 1000, 2048])
def test_position_vectors(width):
    from sleuth_b200.parts.ends import sinusoid_turns
    positions = [0, 1, 2, 63, 64, 1000, 16383, 131071, (1 << 20) - 1]
    torch.testing.assert_close(place_vectors_at([0, 1, 2], width), plain.place_vectors(3, width, torch.float64))
    x0 = torch.randn(len(positions), width, generator=torch.Generator().manual_seed(width))
    x = x0.clone().to(DEV)
    ops().sinusoid_add(x, i32(positions), sinusoid_turns(width, 10000.0, DEV))
    torch.testing.assert_close(x.cpu().double(), x0.double() + place_vectors_at(positions, width), rtol=0, atol=2e-6)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("width", [75, 384])
@pytest.mark.parametrize("one_pass", [True, False])
def test_token_row_pair_row_and_position_vector(one_pass, width, dtype):
    """Portions of unequal lengths, one sequence after another in a slot of its own, the previous token kept between steps."""
    from sleuth_b200.parts.ends import sinusoid_turns
    o = ops()
    g = torch.Generator().manual_seed(width)
    vocab, buckets, mp, mc = 300, 101, 7, 13
    table = torch.randn(vocab, width, generator=g).to(DT[dtype])
    pairs = torch.randn(buckets + 1, width, generator=g).to(DT[dtype])
    w = {"embed": table.double(), "bigram": pairs.double()}
    e = {"scale": 3.0, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}
    seqs = [torch.randint(0, vocab, (n,), generator=g).tolist() for n in (9, 70, 4)]
    slots, turns = [4, 0, 2], sinusoid_turns(width, 10000.0, DEV)
    last = torch.full((6, 1), -1, dtype=torch.int32, device=DEV)
    done, got = [0, 0, 0], [[], [], []]
    for step in ([4, 1, 2], [1, 60, 2], [4, 9, 0]):
        live = [k for k in range(3) if step[k]]
        ids = sum((seqs[k][done[k]:done[k] + step[k]] for k in live), [])
        c = [step[k] for k in live]
        tok_seq = i32(sum(([n] * m for n, m in enumerate(c)), []))
        tok_pos = i32(sum((list(range(done[k], done[k] + step[k])) for k in live), []))
        x = torch.empty(len(ids), width, device=DEV)
        starts, now = i32([0, *np.cumsum(c).tolist()]), i32([slots[k] for k in live])
        if not one_pass:
            o.embed(i32(ids), table.to(DEV), x, 3.0)
        o.pair_embed(i32(ids), None, pairs.to(DEV), x, tok_seq, tok_pos, starts, now, last, vocab, buckets, mp, mc,
                     table=table.to(DEV) if one_pass else None, scale=3.0, turns=turns)
        at = 0
        for k in live:
            got[k].append(x[at:at + step[k]].cpu().double())
            at += step[k]
            done[k] += step[k]
    for k in range(3):
        torch.testing.assert_close(torch.cat(got[k]), plain.embedding(torch.tensor(seqs[k]), w, e), rtol=1e-6, atol=2e-6)
    assert last.view(-1).cpu().tolist() == [seqs[1][-1], -1, seqs[2][-1], -1, seqs[0][-1], -1]


# ---- gains stored less one ----
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("d", [75, 384])
def test_a_norm_whose_gain_is_stored_less_one(d, dtype):
    from sleuth_b200.parts.base import BuildContext, build_norm
    from sleuth_b200.parts.spec import NormSpec
    x, gain = torch.randn(7, d), torch.randn(d) * 0.5
    n = build_norm(NormSpec(d, 1e-3, gain_offset=1.0), BuildContext(torch.device(DEV), DT[dtype], 8))
    n.bind({"weight": gain.to(DEV)})
    out = torch.empty(7, d, dtype=DT[dtype], device=DEV)
    n.forward(x.to(DEV), out)
    torch.testing.assert_close(out.cpu().double(), plain.centred_norm(x.double(), gain.double(), 1e-3), **TOL[dtype])


# ---- attention over the latent cache ----
def paged(rows_per_seq, width, dtype, seed):
    """A pool whose pages are handed out in a scrambled order, and the block table of the sequences."""
    n_pages = sum(-(-len(r) // 64) for r in rows_per_seq) + 3
    order = np.random.default_rng(seed).permutation(n_pages)
    pool = torch.full((n_pages, 64, width), 7.0, dtype=dtype, device=DEV)      # stale contents must never be read
    stride = max(-(-len(r) // 64) for r in rows_per_seq) + 1
    table = torch.full((len(rows_per_seq), stride), -1, dtype=torch.int32)
    k = 0
    for s, rows in enumerate(rows_per_seq):
        for p in range(-(-len(rows) // 64)):
            table[s, p] = int(order[k])
            part = rows[p * 64:(p + 1) * 64]
            pool[order[k], :len(part)] = part.to(dtype).to(DEV)
            k += 1
    return pool, table.to(DEV)


def case(H, dn, dv, R, lengths, seed, loud=()):
    """Random latents, queries and up-projections. ``loud``: (sequence, query position, key position) triples whose score
    is made to stand out, so that a key that is skipped or read from a wrong row changes the result."""
    g = torch.Generator().manual_seed(seed)
    w_uk = torch.randn(H * dn, R, generator=g, dtype=torch.float64) / R ** 0.5
    w_uv = torch.randn(H * dv, R, generator=g, dtype=torch.float64) / R ** 0.5
    seqs = [dict(c=torch.randn(n, R, generator=g, dtype=torch.float64), q=torch.randn(n, H, dn, generator=g, dtype=torch.float64))
            for n in lengths]
    for s, qi, ki in loud:
        k = (seqs[s]["c"][ki] @ w_uk.T).reshape(H, dn)
        seqs[s]["q"][qi] = 12.0 * k / k.norm(dim=-1, keepdim=True)
    return w_uk, w_uv, seqs


def sinks_for(H, kind):
    if kind == "near":          # of the size of the scores: each head's differs
        return torch.linspace(-1.0, 3.0, H, dtype=torch.float64) if H > 1 else torch.tensor([1.0], dtype=torch.float64)
    return torch.full((H,), {"low": -60.0, "high": 40.0}[kind], dtype=torch.float64)


def run(H, dn, dv, R, pasts, counts, dtype, seed, sinks="near", loud=(), splits=1, scale=0.3, general=False):
    o, dt = ops(), DT[dtype]
    lengths = [p + c for p, c in zip(pasts, counts)]
    w_uk, w_uv, seqs = case(H, dn, dv, R, lengths, seed, loud)
    if dtype == "bf16":     # both sides see the same rounded inputs
        for s in seqs:
            s["c"], s["q"] = s["c"].to(dt).double(), s["q"].to(dt).double()
    sink = sinks_for(H, sinks) if sinks else None
    pool, table = paged([s["c"] for s in seqs], R, dt, seed)
    T = sum(counts)
    q = torch.cat([s["q"][p:p + c] for s, p, c in zip(seqs, pasts, counts)])
    q_lat = torch.einsum("thd,hdr->htr", q, w_uk.reshape(H, dn, R)).to(dt).to(DEV).contiguous()
    out = torch.empty(H, T, R, dtype=dt, device=DEV)
    scratch = torch.empty(max(1, o.latent_scratch_floats(T, H, R, splits)), dtype=torch.float32, device=DEV)
    o.latent_attention_general_only(general)
    try:
        o.latent_attention(q_lat, q.to(dt).to(DEV).contiguous(), pool, out, None, None, i32([0, *np.cumsum(counts).tolist()]), i32(pasts),
                           i32(counts), table, max(counts), H, R, 0, dn, 0, 0, scale, splits, scratch,
                           sinks=None if sink is None else sink.float().to(DEV))
        got = torch.einsum("htr,hvr->thv", out.cpu().double(), w_uv.reshape(H, dv, R))
    finally:
        o.latent_attention_general_only(False)
    none = torch.full((H,), -1e9, dtype=torch.float64)
    want = []
    for s, p in zip(seqs, pasts):
        n = len(s["c"])
        k, v = (s["c"] @ w_uk.T).reshape(n, H, dn), (s["c"] @ w_uv.T).reshape(n, H, dv)
        want.append(plain.causal_sink_attention(s["q"], k, v, scale, none if sink is None else sink)[p:])
    return got, torch.cat(want)


SIZES = [(3, 12, 20, 36), (8, 48, 64, 112), (1, 8, 8, 7), (40, 8, 8, 32), (5, 16, 16, 512), (70, 8, 8, 48), (16, 24, 16, 256),
         (20, 16, 16, 272), (33, 8, 8, 64), (2, 16, 16, 528)]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("H, dn, dv, R", SIZES)
def test_attention_with_sinks_prompts(H, dn, dv, R, dtype):
    got, want = run(H, dn, dv, R, pasts=[0, 0, 0, 0, 70], counts=[1, 65, 130, 17, 9], dtype=dtype, seed=H)
    torch.testing.assert_close(got, want, **TOL[dtype])


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("splits", [1, 2, 7])
@pytest.mark.parametrize("H, dn, dv, R", SIZES)
def test_attention_with_sinks_single_tokens(H, dn, dv, R, splits, dtype):
    """One token a sequence: the first of all, one that ends a page, one that begins one, far along; the far ones asking for
    the first token, a page's last row and a page's first row."""
    pasts = [0, 63, 64, 300, 447, 200]
    loud = [(1, 63, 0), (2, 64, 63), (3, 300, 64), (4, 447, 1), (5, 200, 191)]
    got, want = run(H, dn, dv, R, pasts, [1] * 6, dtype, seed=H + 1, loud=loud, splits=splits)
    torch.testing.assert_close(got, want, **TOL[dtype])
    assert float(want.abs().max()) > 0.5         # the loud keys carry the result


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("general", [False, True])
@pytest.mark.parametrize("counts, splits", [([1, 1, 1], 1), ([1, 1, 1], 5), ([33, 2, 65], 1), ([33, 2, 65], 3)])
def test_the_sink_counts_once_and_is_not_scaled(counts, splits, general, dtype):
    """A sink far below the scores is no sink; one far above takes everything; one between shares, the same whatever the
    number of slices and the kernel."""
    pasts = [200, 0, 64]
    args = dict(H=6, dn=16, dv=16, R=64, pasts=pasts, counts=counts, dtype=dtype, seed=3, splits=splits, general=general)
    bare = run(sinks=None, **args)[0]
    torch.testing.assert_close(run(sinks="low", **args)[0], bare, rtol=1e-5, atol=1e-5)
    assert float(run(sinks="high", **args)[0].abs().max()) < 1e-6
    got, want = run(sinks="near", **args)
    torch.testing.assert_close(got, want, **TOL[dtype])
    assert float((got - bare).abs().max()) > 0.1


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_attention_finds_far_keys_and_keys_at_page_borders(dtype):
    loud = [(0, 299, 0), (0, 298, 63), (0, 297, 64), (0, 296, 127), (0, 295, 128), (0, 290, 5), (1, 200, 200), (1, 199, 191),
            (2, 640, 1), (3, 130, 64), (4, 450, 3)]
    pasts, counts = [250, 0, 640, 130, 450], [50, 201, 1, 1, 1]
    got, want = run(4, 16, 12, 48, pasts, counts, dtype, seed=9, loud=loud)
    torch.testing.assert_close(got, want, **TOL[dtype])
    assert float(want.abs().max()) > 0.5


# ---- whole prompts with per-head keys and values ----
PROMPTS = [1, 65, 300, 64, 128, 191]
LOUD = [(1, 64, 0), (1, 63, 62), (2, 299, 0), (2, 298, 63), (2, 297, 64), (2, 200, 128), (3, 63, 1), (4, 127, 0), (5, 190, 64)]


@pytest.mark.parametrize("sinks", ["near", "low", "high"])
@pytest.mark.parametrize("H, dn, dv, R", [(3, 16, 16, 40), (8, 48, 64, 80), (2, 128, 128, 72), (5, 32, 48, 24)])
def test_whole_prompts_on_the_warp_level_kernel(H, dn, dv, R, sinks):
    o, dt = ops(), torch.bfloat16
    w_uk, w_uv, seqs = case(H, dn, dv, R, PROMPTS, seed=H + dn, loud=LOUD)
    T, scale, sink = sum(PROMPTS), 0.3, sinks_for(H, sinks)
    q = torch.cat([s["q"] for s in seqs]).to(dt)
    c = torch.cat([s["c"] for s in seqs])
    kv = torch.cat([c @ w_uk.T, c @ w_uv.T], dim=-1).to(dt)
    out = torch.empty(H, T, dv, dtype=dt, device=DEV)
    starts = [0, *np.cumsum(PROMPTS).tolist()]
    o.head_prompt_attention(q.to(DEV), kv.to(DEV), torch.empty(T, 0, dtype=dt, device=DEV), out, None, None, i32(starts), i32(PROMPTS),
                            max(PROMPTS), H, dn, 0, dv, 0, 0, scale, sinks=sink.float().to(DEV))
    want = torch.cat([plain.causal_sink_attention(q[a:b].double(), kv[a:b, :H * dn].double().reshape(b - a, H, dn),
                                                  kv[a:b, H * dn:].double().reshape(b - a, H, dv), scale, sink)
                      for a, b in zip(starts, starts[1:])])
    torch.testing.assert_close(out.cpu().double().transpose(0, 1), want, **TOL["bf16"])


@pytest.mark.parametrize("lengths", [PROMPTS, [128], [1000, 3], [64, 64, 64, 256], [2, 1, 1, 130, 63]])
@pytest.mark.parametrize("H, d, R", [(5, 64, 128), (3, 128, 272), (1, 64, 8), (16, 128, 64)])
def test_whole_prompts_on_the_tensor_memory_kernel(H, d, R, lengths):
    """Latents normed, keys and values formed into pages of the step's own, attention read from those pages: the pages' table,
    the cleared rows behind every sequence's end (scratch memory full of NaN before), sinks, loud keys."""
    o, dt = ops(), torch.bfloat16
    loud = [(s, i, j) for s, i, j in LOUD if lengths is PROMPTS]
    w_uk, w_uv, seqs = case(H, d, d, R, lengths, seed=H + d, loud=loud)
    T, n, scale, sink = sum(lengths), len(lengths), 0.3, sinks_for(H, "near")
    starts = [0, *np.cumsum(lengths).tolist()]
    q = torch.cat([s["q"] for s in seqs]).to(dt)
    lat = torch.cat([s["c"] for s in seqs]).float()
    gain = 1.0 + 0.2 * torch.randn(R, generator=torch.Generator().manual_seed(R))
    n_pages = o.prompt_pages(T, n)
    k_pages, v_pages = (torch.full((n_pages, H, 64, d), float("nan"), dtype=dt, device=DEV) for _ in range(2))
    table = torch.full((n, -(-max(lengths) // 64)), -1, dtype=torch.int32, device=DEV)
    tok_seq = i32(sum(([s] * m for s, m in enumerate(lengths)), []))
    tok_pos = i32(sum((list(range(m)) for m in lengths), []))
    c_out, k_out = torch.empty(T, R, dtype=dt, device=DEV), torch.empty(T, 0, dtype=dt, device=DEV)
    o.latent_post(lat.to(DEV), None, gain.to(DEV), None, None, None, None, tok_seq, tok_pos, None, 0, R, 0, 0, 1e-5, c_out=c_out,
                  k_out=k_out, dtype=dt, pages=(table, i32(starts), v_pages))
    torch.testing.assert_close(c_out.cpu().double(), plain.rms(lat.double(), 1e-5) * gain.double(), **TOL["bf16"])
    pages = [table[s, p].item() for s, m in enumerate(lengths) for p in range(-(-m // 64))]
    assert len(set(pages)) == len(pages) and min(pages) >= 0 and max(pages) < n_pages
    w = torch.cat([w_uk, w_uv]).to(dt)
    o.gemm_tc_qkv(c_out, w.to(DEV), 0, H, d, None, None, None, None, None, 1e-6, None, k_pages, v_pages, tok_seq, tok_pos, table)
    c = c_out.cpu().double()
    kv = (c @ w.double().T).to(dt)
    for s, m in enumerate(lengths):       # the pages hold every head's rows, and zeros behind the last value row
        for p in range(-(-m // 64)):
            page, rows = table[s, p].item(), min(64, m - 64 * p)
            mine = kv[starts[s] + 64 * p:starts[s] + 64 * p + rows].double()
            torch.testing.assert_close(k_pages[page, :, :rows].cpu().double().transpose(0, 1), mine[:, :H * d].reshape(rows, H, d), rtol=1e-2, atol=1e-2)
            torch.testing.assert_close(v_pages[page, :, :rows].cpu().double().transpose(0, 1), mine[:, H * d:].reshape(rows, H, d), rtol=1e-2, atol=1e-2)
            assert bool((v_pages[page, :, rows:] == 0).all())
    for wide in (None, False, True):
        y = torch.empty(T, H * d, dtype=dt, device=DEV)
        o.attention_tc(q.to(DEV), k_pages, v_pages, y, i32(starts), i32([0] * n), i32(lengths), table, max(lengths), H, H, d, 0, scale,
                       max_keys=max(lengths), sinks=sink.float().to(DEV), wide=wide)
        torch.cuda.synchronize()
        o.gemm_tc_check(torch.device(DEV))
        want = torch.cat([plain.causal_sink_attention(q[a:b].double(), kv[a:b, :H * d].double().reshape(b - a, H, d),
                                                      kv[a:b, H * d:].double().reshape(b - a, H, d), scale, sink)
                          for a, b in zip(starts, starts[1:])])
        torch.testing.assert_close(y.view(T, H, d).cpu().double(), want, **TOL["bf16"])


# ---- the output gate ----
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("T, N, K", [(3, 60, 75), (40, 96, 64), (130, 320, 128), (300, 72, 104), (257, 1000, 192), (4100, 256, 64)])
def test_gate_in_the_products_epilogue(T, N, K, dtype):
    from sleuth_b200.parts.base import Workspace
    from sleuth_b200.parts.linear import Linear
    g = torch.Generator().manual_seed(T)
    h, w, val = torch.randn(T, K, generator=g), torch.randn(N, K, generator=g) * (3.0 / K ** 0.5), torch.randn(T, N, generator=g)
    h, w, val = (t.to(DT[dtype]) for t in (h, w, val))
    y = val.clone().to(DEV)
    Linear(w.to(DEV), DT[dtype]).gate_values(h.to(DEV), y, ws=Workspace(DEV))
    torch.cuda.synchronize()
    ops().gemm_tc_check(torch.device(DEV))
    torch.testing.assert_close(y.cpu().double(), val.double() * torch.sigmoid(h.double() @ w.double().T), **TOL[dtype])


# ---- the router ----
@pytest.mark.parametrize("T", [1, 9, 300])
@pytest.mark.parametrize("E, top, d", [(8, 3, 96), (12, 12, 64), (70, 2, 128)])
def test_router_bias_joins_logits_that_a_product_formed(T, E, top, d):
    o = ops()
    g = torch.Generator().manual_seed(T + E)
    h = torch.randn(T, d, generator=g).to(torch.bfloat16)
    w = {"router": torch.randn(E, d, generator=g).to(torch.bfloat16).double(), "router.b": 5.0 * torch.randn(E, generator=g).double()}
    idx, wt, margin = plain.expert_choice(h.double(), w, "", {"router": {"experts": E, "top": top}})
    z = (h.double() @ w["router"].T).float().to(DEV).contiguous()
    choice, rank, place, order = (torch.empty(T * top, dtype=torch.int32, device=DEV) for _ in range(4))
    weight, counts = torch.empty(T * top, device=DEV), torch.empty(E, dtype=torch.int32, device=DEV)
    o.moe_route(h.to(DEV), w["router"].float().to(DEV), w["router.b"].float().to(DEV), choice, weight, rank, counts, place, order, top,
                logits=z, logits_ready=True)
    clear = margin > 1e-4
    assert torch.equal(choice.cpu().view(T, top).long()[clear], idx[clear]) and int(clear.sum()) >= T - 1
    torch.testing.assert_close(weight.cpu().view(T, top).double()[clear], wt[clear], rtol=1e-4, atol=2e-5)
    # the bias decides some of the choices
    bare, _, _ = plain.expert_choice(h.double(), {**w, "router.b": w["router.b"] * 0}, "", {"router": {"experts": E, "top": top}})
    assert top == E or T < 9 or not torch.equal(bare, idx)


# ---- single-token steps of few sequences ----
def turned(v, positions, dims, base=500.0):
    """The first ``dims`` channels of the last axis turned, channel i with i + dims / 2, by position * base^(-2i / dims)."""
    if not dims:
        return v
    half = dims // 2
    ang = positions.double()[:, None] * base ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)[None, :]
    shape = [v.shape[0]] + [1] * (v.dim() - 2) + [half]
    c, s = ang.cos().reshape(shape), ang.sin().reshape(shape)
    a, b = v[..., :half], v[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, v[..., dims:]], dim=-1)


def turn_tables(count, dims, base=500.0):
    ang = torch.arange(count, dtype=torch.float64)[:, None] * base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)[None, :]
    return ang.cos().float().to(DEV), ang.sin().float().to(DEV)


@pytest.mark.parametrize("splits", [1, 2, 7, 64])
@pytest.mark.parametrize("H, R, P, window", [(1, 16, 0, 0), (6, 64, 0, 0), (16, 512, 0, 0), (16, 256, 32, 0), (20, 272, 0, 0), (33, 112, 16, 100),
                                             (70, 48, 0, 0), (16, 512, 64, 130), (5, 144, 16, 1), (64, 512, 0, 64)])
def test_attention_of_single_tokens(H, R, P, window, splits):
    """Scores, softmax and weighted sum over scattered pages, with sinks (joined in the kernel, or with the slices), windows,
    a rotated part; the first token of all, a page's last and first places, far keys that stand out."""
    o, dt = ops(), torch.bfloat16
    g = torch.Generator().manual_seed(H + R)
    pasts = [0, 63, 64, 300, 447, 200, 128]
    loud = {1: 0, 2: 63, 3: 64, 4: 1, 5: 191, 6: 127}
    n, scale, sink = len(pasts), 0.25, sinks_for(H, "near")
    w_v = torch.randn(H, 8, R, generator=g, dtype=torch.float64) / R ** 0.5
    rows = [torch.randn(p + 1, R + P, generator=g).to(dt).double() * 0.5 for p in pasts]
    q = torch.randn(n, H, R + P, generator=g, dtype=torch.float64)
    for s, k in loud.items():
        key = turned(rows[s][:, R:], torch.arange(len(rows[s])), P)[k] if P else rows[s][k, :0]
        near = torch.cat([rows[s][k, :R], turned(key[None], torch.tensor([-pasts[s]]), P)[0]]) if P else rows[s][k]
        q[s] = 30.0 * near / near.norm()
    q = q.to(dt).double()
    cached = [torch.cat([r[:, :R], turned(r[:, R:], torch.arange(len(r)), P)], -1).to(dt).double() for r in rows]
    pool, table = paged(cached, R + P, dt, H)
    cos, sin = turn_tables(512, P) if P else (None, None)
    q_raw = torch.cat([torch.randn(n, H, 8, generator=g, dtype=torch.float64), q[..., R:]], -1).to(dt).to(DEV).contiguous()
    q_lat = q[..., :R].permute(1, 0, 2).to(dt).to(DEV).contiguous()
    parts = torch.full((max(1, o.latent_scratch_floats(n, H, R, splits)),), float("nan"), device=DEV)
    out = torch.empty(H, n, R, dtype=dt, device=DEV)
    assert o.latent_decode_supported(H, R, P, 32, 32, dt) == (R % 32 == 0)
    sinks = sink.float().to(DEV)
    o.latent_decode_attention(q_lat, q_raw if P else None, pool, out if splits == 1 else None, parts, cos, sin, i32(pasts), table, R, P, 8, P,
                              window, scale, splits, sinks=sinks)
    want = []
    for s, p in enumerate(pasts):
        lo = max(0, p - window + 1) if window else 0
        k = cached[s][lo:].unsqueeze(1).expand(-1, H, -1)
        qq = torch.cat([q[s, :, :R], turned(q[s, :, R:][None], torch.tensor([p]), P)[0].to(dt).double()], -1)
        sc = torch.einsum("hd,jhd->hj", qq, k) * scale
        pr = plain.sink_softmax(sc[:, None, :], sink)[:, 0]
        want.append(torch.einsum("hj,jr->hr", pr, cached[s][lo:, :R]))
    want = torch.stack(want, 1)
    if splits == 1:
        got = out.cpu().double()
    else:       # the slices as they are defined: sums, maxima and masses; an empty slice has mass 0
        pt = parts.cpu().double().view(splits, n, H, R + 2)
        m, mass = pt[..., R], pt[..., R + 1]
        top = torch.maximum(m.amax(0), sink[None, :])
        f = torch.where(mass > 0, torch.exp(m - top), torch.zeros_like(m))
        total = (f * mass).sum(0) + torch.exp(sink[None, :] - top)
        got = (torch.where((mass > 0)[..., None], pt[..., :R], torch.zeros_like(pt[..., :R])) * f[..., None]).sum(0) / total[..., None]
        got = got.permute(1, 0, 2)
    torch.testing.assert_close(got, want, rtol=2e-2, atol=1e-2)
    if splits == 1 or R % 32:
        return
    # and joined, up-projected and gated (R a multiple of 32)
    dv = 24
    w = (torch.randn(H, dv, R, generator=g) / R ** 0.5).to(dt)
    gate = 2.0 * torch.randn(n, 3 + H * dv, generator=g)
    for view, per in ((gate[:, 3:], False), (gate[:, 3:3 + H], True), (None, False)):
        y = torch.empty(n, H * dv, dtype=dt, device=DEV)
        o.latent_value(parts, None, w.to(DEV), None if view is None else gate.to(DEV)[:, 3:3 + view.shape[1]], y, splits, sinks=sinks)
        val = torch.einsum("hnr,hjr->nhj", want, w.double())
        if view is not None:
            z = torch.sigmoid(view.double())
            val = val * (z[:, :, None] if per else z.reshape(n, H, dv))
        torch.testing.assert_close(y.cpu().double(), val.reshape(n, -1), rtol=2e-2, atol=1e-2)


@pytest.mark.parametrize("n", [1, 8, 9, 20])
@pytest.mark.parametrize("H, dn, dv, R, P, q_rank", [(3, 32, 20, 64, 0, 96), (16, 64, 64, 256, 0, 384), (5, 96, 128, 96, 0, 32), (1, 32, 8, 32, 8, 64),
                                                    (4, 128, 256, 512, 64, 0), (2, 160, 40, 1024, 16, 1536)])
def test_queries_and_values_of_single_tokens(n, H, dn, dv, R, P, q_rank):
    """Norms, both steps of the queries, the cache rows and nothing else in the pool; finished sums up-projected and gated."""
    o, dt = ops(), torch.bfloat16
    g = torch.Generator().manual_seed(n + R)
    K = q_rank or 128
    lat = torch.randn(n, q_rank + R + P + 11, generator=g)
    h = torch.randn(n, K, generator=g).to(dt)
    qg, cg = 1 + 0.2 * torch.randn(K, generator=g), 1 + 0.2 * torch.randn(R, generator=g)
    w_uq = (torch.randn(H * (dn + P), K, generator=g) / K ** 0.5).to(dt)
    w_uk = (torch.randn(H, dn, R, generator=g) / dn ** 0.5).to(dt)
    pasts = [int(v) for v in torch.randint(0, 130, (n,), generator=g)]
    pool, table = paged([torch.zeros(p + 1, R + P) for p in pasts], R + P, dt, n)
    before = pool.clone()
    cos, sin = turn_tables(140, P) if P else (None, None)
    q_lat = torch.full((H, n, R), float("nan"), dtype=dt, device=DEV)
    q_raw = torch.zeros(n, H, dn + P, dtype=dt, device=DEV) if P else None
    assert o.latent_decode_supported(H, R, P, K, dn, dt) == (R <= 512 and (R + P) % 16 == 0)
    o.latent_query(lat.to(DEV), qg.to(DEV) if q_rank else None, cg.to(DEV), None if q_rank else h.to(DEV), w_uq.to(DEV),
                   w_uk.transpose(1, 2).contiguous().to(DEV), cos, sin, q_lat, q_raw, pool, i32(pasts), table, q_rank, R, P, dn, P, 1e-5)
    x = (plain.rms(lat[:, :q_rank].double(), 1e-5) * qg.double()).to(dt).double() if q_rank else h.double()
    q = (x @ w_uq.double().T).reshape(n, H, dn + P)
    torch.testing.assert_close(q_lat.cpu().double(), torch.einsum("nhd,hdr->hnr", q[..., :dn].to(dt).double(), w_uk.double()), rtol=2e-2, atol=2e-2)
    if P:
        torch.testing.assert_close(q_raw[..., dn:].cpu().double(), q[..., dn:], rtol=1e-2, atol=1e-2)
    want = torch.cat([plain.rms(lat[:, q_rank:q_rank + R].double(), 1e-5) * cg.double(),
                      turned(lat[:, q_rank + R:q_rank + R + P].double(), torch.tensor(pasts), P)], -1)
    for t, p in enumerate(pasts):
        at = (table[t, p // 64].item(), p % 64)
        torch.testing.assert_close(pool[at].cpu().double(), want[t], rtol=1e-2, atol=1e-2)
        before[at] = pool[at]
    assert torch.equal(pool, before)
    o_lat = torch.randn(H, n, R, generator=g).to(dt)
    w_uv = (torch.randn(H, dv, R, generator=g) / R ** 0.5).to(dt)
    gate = 2.0 * torch.randn(n, 5 + H * dv, generator=g)
    y = torch.empty(n, H * dv, dtype=dt, device=DEV)
    o.latent_value(None, o_lat.to(DEV), w_uv.to(DEV), gate.to(DEV)[:, 5:], y, 1)
    val = torch.einsum("hnr,hjr->nhj", o_lat.double(), w_uv.double()).reshape(n, -1) * torch.sigmoid(gate[:, 5:].double())
    torch.testing.assert_close(y.cpu().double(), val, rtol=2e-2, atol=1e-2)


def test_the_slices_follow_the_batch_and_the_longest_sequence():
    o = ops()
    one = o.latent_decode_splits(1, 16, 256, 0, 64 * 20)
    assert one == 20 and o.latent_decode_splits(1, 16, 256, 0, 64) == 1 and o.latent_decode_splits(1000, 16, 256, 0, 4096) == 1
    assert 1 < o.latent_decode_splits(8, 16, 512, 0, 4096) <= 64
    assert not o.latent_decode_supported(16, 528, 0, 64, 64, torch.bfloat16) and not o.latent_decode_supported(16, 256, 0, 64, 64, torch.float32)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("T, top", [(1, 3), (5, 2)])
def test_further_rows_join_the_experts_sum(T, top, dtype):
    """The rows of a shared expert that ran beside the router are added by the experts' last kernel."""
    o, dt = ops(), DT[dtype]
    g = torch.Generator().manual_seed(T)
    E, d, ff = 6, 72, 40
    h = torch.randn(T, d, generator=g).to(dt)
    gu, dn = (torch.randn(E, 2 * ff, d, generator=g) / d ** 0.5).to(dt), (torch.randn(E, d, ff, generator=g) / ff ** 0.5).to(dt)
    choice = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).view(-1)
    weight, x, extra = torch.rand(T * top, generator=g), torch.randn(T, d, generator=g), torch.randn(T, d, generator=g)
    junk = torch.zeros(max(E, T * top), dtype=torch.int32, device=DEV)
    got = []
    for more in (None, extra.to(DEV)):
        y = x.clone().to(DEV)
        o.moe_experts(h.to(DEV), gu.to(DEV), dn.to(DEV), junk, junk, weight.to(DEV), torch.empty(T * top, ff, dtype=dt, device=DEV),
                      torch.empty(T * top, d, device=DEV), y, top, choice=choice.int().to(DEV), extra=more)
        got.append(y.cpu())
    torch.testing.assert_close(got[1], got[0] + extra, rtol=1e-5, atol=1e-5)
    want = x.double()
    for p, e in enumerate(choice.tolist()):
        w = {"gate": gu[e, :ff].double(), "up": gu[e, ff:].double(), "down": dn[e].double()}
        want[p // top] += weight[p].double() * plain.gated_mlp(h[p // top:p // top + 1].double(), w, "")[0]
    torch.testing.assert_close(got[0].double(), want, **TOL[dtype])
    with pytest.raises(Exception):
        o.moe_experts(h.to(DEV), gu.to(DEV), dn.to(DEV), junk, junk, weight.to(DEV), torch.empty(T * top, ff, dtype=dt, device=DEV),
                      torch.empty(T * top, d, device=DEV), x.to(DEV), top, choice=choice.int().to(DEV), extra=extra[:, :8].to(DEV))
