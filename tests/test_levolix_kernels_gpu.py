"""Each kernel that came with the Levolix design, or learned something for it, beside its plain function: the recurrences with one
decay a head (token by token, in chunks, and a whole single-token step), their preparation, attention inside chunks of positions
with a one in the denominator (a loud key at a chunk's first position and just in front of it, in prompts, portions and single
tokens, on every attention kernel), biases in the post-processing of projections, the closing norm that joins two results and
leaves the rounded stream, and experts that return their input."""

from __future__ import annotations

import pytest
import torch

from plain import levolix_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def ops():
    from sleuth_b200.kernels import ops as o
    return o


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def batch_tables(counts, pasts=None):
    """tok_seq, tok_pos, seq_start for sequences that bring ``counts`` tokens behind ``pasts`` earlier ones."""
    pasts = pasts or [0] * len(counts)
    seq = [s for s, c in enumerate(counts) for _ in range(c)]
    pos = [p + i for c, p in zip(counts, pasts) for i in range(c)]
    start = [0]
    for c in counts:
        start.append(start[-1] + c)
    return i32(seq), i32(pos), i32(start)


# ---------------------------------------------------------------- recurrences ----

def scan_case(H, G, N, P, delta, lengths, cuts, seed=0, decay=None, make=None):
    """Runs ``lengths`` sequences through ``state_scan`` in the portions ``cuts`` (the last one takes the rest) and compares
    outputs and last states with the plain loop; slots of other sequences must stay as they are."""
    o = ops()
    g = torch.Generator().manual_seed(seed + H * 1000 + N)
    n_slots = len(lengths) + 3
    slots = torch.randperm(n_slots, generator=g)[:len(lengths)].tolist()
    others = [s for s in range(n_slots) if s not in slots]
    data = []
    for n in lengths:
        q, k = plain.unit(torch.randn(n, G, N, generator=g)), plain.unit(torch.randn(n, G, N, generator=g))
        v = torch.randn(n, H, P, generator=g)
        logd = -torch.rand(n, H, generator=g) * 0.2 if decay is None else decay.log().expand(n, H)
        beta = torch.rand(n, H, generator=g)
        if make is not None:
            make(q, k, v, logd, beta)
        data.append((q, k, v, logd, beta))
    want = []
    for q, k, v, logd, beta in data:
        qq, kk = (t.repeat_interleave(H // G, dim=1).double() for t in (q, k))
        if delta:
            out, S = plain.delta_recurrence(logd.double().exp(), beta.double(), kk, v.double(), qq)
        else:
            out, S = plain.decayed_recurrence(decay.double(), kk, v.double(), qq)
        want.append((out.reshape(len(q), H * P), S))
    for cut_list in cuts:
        state = torch.full((n_slots, H, N, P), 3.0, device=DEV)
        state[slots] = 0.0
        done, got = [0] * len(lengths), [[] for _ in lengths]
        for cut in [*cut_list, None]:
            take = [n - d if cut is None else min(cut, n - d) for n, d in zip(lengths, done)]
            live = [i for i, t in enumerate(take) if t > 0]
            if not live:
                continue
            part = [torch.cat([data[i][j][done[i]:done[i] + take[i]].reshape(take[i], -1) for i in live]).to(DEV) for j in range(5)]
            qkv = torch.cat([part[0], part[1], part[2], torch.full((part[0].shape[0], 3), 9.0, device=DEV)], dim=1)     # views of wider rows
            _, _, start = batch_tables([take[i] for i in live])
            longest = max(take[i] for i in live)
            need = o.state_scan_scratch_floats(len(live), longest, H, N, P, delta)
            assert (need > 0) == (longest > 24 and N <= 128)
            scratch = torch.full((need,), float("nan"), device=DEV) if need else None
            out = torch.full((qkv.shape[0], H * P), float("nan"), device=DEV)
            o.state_scan(qkv[:, :G * N], qkv[:, G * N:2 * G * N], qkv[:, 2 * G * N:2 * G * N + H * P],
                         part[3] if decay is None else decay.log().to(DEV), state, i32([slots[i] for i in live]), start, out, H, G,
                         longest, beta=part[4] if delta else None, scratch=scratch)
            at = 0
            for i in live:
                got[i].append(out[at:at + take[i]].cpu())
                at += take[i]
                done[i] += take[i]
        for i in range(len(lengths)):
            torch.testing.assert_close(torch.cat(got[i]).double(), want[i][0], rtol=1e-4, atol=1e-4)
            torch.testing.assert_close(state[slots[i]].cpu().double(), want[i][1], rtol=1e-4, atol=1e-4)
        assert bool((state[others] == 3.0).all())


SIZES = [(3, 1, 12, 16), (4, 4, 40, 10), (2, 2, 72, 33), (1, 1, 128, 130), (6, 3, 64, 64), (2, 1, 96, 5), (2, 1, 33, 70), (1, 1, 136, 20)]


@pytest.mark.parametrize("H,G,N,P", SIZES)
def test_gated_delta_rule_token_by_token_and_in_chunks(H, G, N, P):
    scan_case(H, G, N, P, True, [1, 150, 7, 64, 65], [[], [3, 1], [70], [25, 33], [64]])


@pytest.mark.parametrize("H,G,N,P", SIZES)
def test_fixed_decay_token_by_token_and_in_chunks(H, G, N, P):
    decay = torch.tensor([0.9995, 0.5, 1.0, 0.0, 0.97, 0.9])[:H]
    scan_case(H, G, N, P, False, [1, 150, 7, 64, 65], [[], [3, 1], [70], [25, 33], [64]], decay=decay)


def test_a_write_is_read_hundreds_of_tokens_later_and_taken_back_by_its_key():
    """One loud value under one key; slow decay; a query with that key far behind still reads it, across many chunks; a later
    write under the same key with full strength replaces it (the delta rule) instead of adding to it."""
    def make(q, k, v, logd, beta):
        n = len(q)
        logd[:] = -1e-4
        if n > 300:
            mark = torch.zeros(k.shape[-1])
            mark[3] = 1.0
            k[..., 3] = 0.0            # nobody else writes along this channel
            q[..., 3] = 0.0
            k[5], v[5], beta[5] = mark, 50.0, 1.0
            q[290] = mark
            k[295], v[295], beta[295] = mark, -20.0, 1.0
            q[n - 1] = mark
    scan_case(2, 1, 64, 32, True, [330, 40], [[], [100, 100], [64, 64, 64, 64, 40]], make=make)


@pytest.mark.parametrize("strength", [0.0, 1.0])
def test_equal_keys_and_extreme_decays(strength):
    """Every token writes under the same key at the ends of the strengths' range; decays from none to complete."""
    def make(q, k, v, logd, beta):
        k[:] = k[0]
        beta[:] = strength
        logd[::7] = -200.0
        logd[1::7] = 0.0
    scan_case(2, 2, 32, 16, True, [200, 64], [[], [64], [90, 30]], make=make)


@pytest.mark.parametrize("N,P,H,G", [(12, 10, 3, 1), (64, 64, 4, 2), (128, 128, 2, 1), (40, 200, 2, 2), (136, 96, 1, 1), (256, 64, 1, 1), (128, 256, 2, 2), (33, 130, 1, 1), (16, 520, 1, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("delta", [True, False])
def test_a_single_token_step_from_the_projections_to_the_gated_heads(N, P, H, G, dtype, delta):
    o = ops()
    if not delta:
        G = H
    if not o.state_token_supported(N, P):
        assert P > 512
        return
    g = torch.Generator().manual_seed(N + P)
    n, eps, T = 3, 1e-5, 4
    slots = [4, 0, 2]
    state = torch.full((6, H, N, P), 2.0, device=DEV)
    state[slots] = 0.0
    rot = 0 if delta else (N // 4) * 2
    decay = torch.tensor([0.99, 0.3, 1.0, 0.0])[:H]
    gain = torch.randn(P, generator=g) + 1 if delta else None
    a_log, dt_bias = torch.randn(H, generator=g), torch.randn(H, generator=g) - 1
    pos0 = [0, 17, 300]
    tol = dict(rtol=2e-4, atol=2e-4) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)
    S = [torch.zeros(H, N, P, dtype=torch.float64) for _ in range(n)]
    i = torch.arange(rot // 2, dtype=torch.float64)
    table = torch.arange(400, dtype=torch.float64)[:, None] * 100.0 ** (-2.0 * i / max(rot, 1))[None]
    cos, sin = table.cos().float().to(DEV), table.sin().float().to(DEV)
    for t in range(T):
        q, k = torch.randn(n, G, N, generator=g), torch.randn(n, G, N, generator=g)
        v, gate = torch.randn(n, H, P, generator=g), torch.randn(n, H * P, generator=g)
        raw = torch.randn(n, 2 * H, generator=g)
        rows = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1), gate, raw], dim=1).to(DEV)
        a, b, c = G * N, 2 * G * N, 2 * G * N + H * P
        out = torch.empty(n, H * P, dtype=dtype, device=DEV)
        kw = dict(q_scale=N ** -0.5, gain=None if gain is None else gain.to(DEV))
        if delta:
            kw.update(raw_beta=rows[:, c + H * P:c + H * P + H], raw_step=rows[:, c + H * P + H:], dt_bias=dt_bias.to(DEV), a_log=a_log.to(DEV), unit_eps=1e-6)
        else:
            kw.update(decay=decay.to(DEV), cos=cos if rot else None, sin=sin if rot else None, tok_pos=i32([p + t for p in pos0]), rot=rot)
        o.state_token(rows[:, :a], rows[:, a:b], rows[:, b:c], rows[:, c:c + H * P], state, i32(slots), out, H, G, eps, **kw)
        for s in range(n):
            qs, ks = q[s].double()[None], k[s].double()[None]
            if delta:
                qs, ks = plain.unit(qs), plain.unit(ks)
                beta = torch.sigmoid(raw[s, :H].double())[None]
                dec = torch.exp(-torch.exp(a_log.double()) * plain.softplus(raw[s, H:].double() + dt_bias.double()))[None]
                want, S[s] = plain.delta_recurrence(dec, beta, ks.repeat_interleave(H // G, 1), v[s].double()[None],
                                                    qs.repeat_interleave(H // G, 1) * N ** -0.5, S[s])
            else:
                ang = plain.angles(torch.tensor([pos0[s] + t]), rot, 100.0, torch.float64)
                qs, ks = plain.rotate_halves(qs, ang), plain.rotate_halves(ks, ang) * N ** -0.5
                want, S[s] = plain.decayed_recurrence(decay.double(), ks, v[s].double()[None], qs, S[s])
            want = plain.head_norm_and_gate(want, None if gain is None else gain.double(), gate[s].double()[None], eps)
            torch.testing.assert_close(out[s].cpu().double(), want[0], **tol)
            scale = 1.0 if delta else N ** 0.5          # the kernel keeps unscaled keys and scales the queries instead
            torch.testing.assert_close(state[slots[s]].cpu().double() / scale, S[s], rtol=2e-4, atol=2e-4)
    assert bool((state[[1, 3, 5]] == 2.0).all())


def test_delta_preparation_and_rotation_in_place():
    o = ops()
    g = torch.Generator().manual_seed(1)
    T, G, N, H = 37, 3, 40, 6
    rows = torch.randn(T, 2 * G * N + 5, generator=g)
    raw = torch.randn(T, 2 * H + 1, generator=g) * 4
    a_log, dt_bias = torch.randn(H, generator=g), torch.randn(H, generator=g)
    dev = rows.to(DEV)
    beta, logd = torch.empty(T, H, device=DEV), torch.empty(T, H, device=DEV)
    r = raw.to(DEV)
    o.delta_prep(dev, r[:, :H], r[:, H:2 * H], dt_bias.to(DEV), a_log.to(DEV), beta, logd, G, N, N ** -0.5, 1e-6)
    u = plain.unit(rows[:, :2 * G * N].double().reshape(T, 2 * G, N))
    u[:, :G] *= N ** -0.5
    torch.testing.assert_close(dev[:, :2 * G * N].cpu().double(), u.reshape(T, -1), rtol=1e-5, atol=1e-6)
    assert torch.equal(dev[:, 2 * G * N:].cpu(), rows[:, 2 * G * N:])
    torch.testing.assert_close(beta.cpu().double(), torch.sigmoid(raw[:, :H].double()), rtol=1e-5, atol=1e-6)
    torch.testing.assert_close(logd.cpu().double(), -torch.exp(a_log.double()) * plain.softplus(raw[:, H:2 * H].double() + dt_bias.double()), rtol=1e-5, atol=1e-6)
    for neighbours, turn in ((False, plain.rotate_halves), (True, plain.rotate_neighbours)):
        for rot in (N, 16, 0):
            pos = torch.randint(0, 900, (T,), generator=g)
            dev = rows.to(DEV)
            i = torch.arange(rot // 2, dtype=torch.float64)
            table = torch.arange(900, dtype=torch.float64)[:, None] * 1000.0 ** (-2.0 * i / max(rot, 1))[None]
            o.rotate_rows(dev, table.cos().float().to(DEV) if rot else None, table.sin().float().to(DEV) if rot else None, pos.to(torch.int32).to(DEV),
                          2 * G, N, rot, neighbours)
            want = turn(rows[:, :2 * G * N].double().reshape(T, 2 * G, N), plain.angles(pos, rot, 1000.0, torch.float64)).reshape(T, -1)
            torch.testing.assert_close(dev[:, :2 * G * N].cpu().double(), want, rtol=1e-5, atol=1e-5)
            assert torch.equal(dev[:, 2 * G * N:].cpu(), rows[:, 2 * G * N:])


# ---------------------------------------------------------------- attention inside chunks ----

def chunk_case(path, dtype, H, G, d, dv, lengths, pasts, size, loud):
    """Queries at positions pasts .. lengths - 1 of each sequence over a paged cache with scattered pages and a one in the
    denominator. ``loud``: the position of a key (or None) that points the way of the sequence's last query."""
    o = ops()
    g = torch.Generator().manual_seed(size * 7 + d)
    n = len(lengths)
    stride = max((L + 63) // 64 for L in lengths) + 1
    pages = n * stride + 2
    perm = torch.randperm(pages, generator=g)[:n * stride].reshape(n, stride)
    k_pool = torch.full((pages, G, 64, d), 7.0, dtype=dtype, device=DEV)       # leftovers of other sequences
    v_pool = torch.full((pages, G, 64, dv), 7.0, dtype=dtype, device=DEV)
    seqs = []
    for s, L in enumerate(lengths):
        q, k, v = torch.randn(L, H, d, generator=g), torch.randn(L, G, d, generator=g), torch.randn(L, G, dv, generator=g)
        if loud is not None and 0 <= loud < L - 1:
            q[L - 1] = 1.0
            k[loud] = 3.0
        q, k, v = (t.to(dtype) for t in (q, k, v))
        seqs.append((q, k, v))
        for j in range(L):
            page = int(perm[s, j // 64])
            k_pool[page, :, j % 64] = k[j].to(DEV)
            v_pool[page, :, j % 64] = v[j].to(DEV)
    table = perm.to(torch.int32)
    spare = next(i for i in range(pages) if i not in set(perm.flatten().tolist()))
    for s, p in enumerate(pasts):          # pages in front of the first query's chunk may hold another sequence by now
        table[s, :p // size * size // 64] = spare
    table = table.to(DEV)
    counts = [L - p for L, p in zip(lengths, pasts)]
    tok_seq, tok_pos, start = batch_tables(counts, pasts)
    q = torch.cat([t[0][p:] for t, p in zip(seqs, pasts)]).contiguous().to(DEV)
    T = q.shape[0]
    out = torch.empty(T, H * dv, dtype=dtype, device=DEV)
    sinks = torch.zeros(H, device=DEV)
    scale = 0.3
    if path == "general":
        o.attention(q, k_pool, v_pool, out, tok_seq, tok_pos, table, H, G, d, -size, scale, sinks=sinks, value_dim=dv)
    elif max(counts) == 1:
        for splits in (1, 3):
            scratch = torch.empty(max(o.decode_scratch_floats(n, H, d, splits), 1), device=DEV)
            o.attention_decode(q, k_pool, v_pool, out, start, i32(pasts), table, H, G, d, -size, scale, splits, scratch, sinks=sinks)
    elif path == "mma":
        o.attention_prefill(q, k_pool, v_pool, out, start, i32(pasts), i32(counts), table, max(counts), H, G, d, -size, scale, sinks=sinks)
    else:
        o.attention_tc(q, k_pool, v_pool, out, start, i32(pasts), i32(counts), table, max(counts), H, G, d, -size, scale, wide=path == "tc_wide",
                       max_keys=max(lengths), sinks=sinks)
        o.gemm_tc_check(torch.device(DEV))
    want = [plain.attend(*(t.double() for t in s), scale, plain.same_chunk(L, size)).reshape(L, -1)[p:] for s, L, p in zip(seqs, lengths, pasts)]
    tol = dict(rtol=2e-4, atol=2e-4) if dtype == torch.float32 else dict(rtol=3e-2, atol=3e-2)
    torch.testing.assert_close(out.cpu().double(), torch.cat(want), **tol)


@pytest.mark.parametrize("path,dtype,H,G,d,dv", [("general", torch.float32, 4, 2, 16, 24), ("general", torch.bfloat16, 3, 1, 24, 40),
                                                 ("mma", torch.bfloat16, 6, 2, 64, 64), ("mma", torch.bfloat16, 4, 4, 128, 128),
                                                 ("tc", torch.bfloat16, 8, 2, 64, 64), ("tc_wide", torch.bfloat16, 8, 2, 64, 64),
                                                 ("tc", torch.bfloat16, 4, 2, 128, 128), ("tc_wide", torch.bfloat16, 2, 2, 128, 128)])
@pytest.mark.parametrize("size", [1, 2, 37, 64, 65, 130, 128])
def test_a_loud_key_at_a_chunks_first_position_and_just_in_front_of_it(path, dtype, H, G, d, dv, size):
    last = 3 * size + size // 2 if size > 30 else 41 * size        # the last query, inside a chunk
    first = last // size * size
    for loud in (first, first - 1):
        L = last + 1
        chunk_case(path, dtype, H, G, d, dv, [L, 200, 3], [0, 0, 0], size, loud)
        chunk_case(path, dtype, H, G, d, dv, [L, 150], [max(0, L - 70), 64], size, loud)
        chunk_case(path, dtype, H, G, d, dv, [L, 200, 3], [L - 1, 199, 2], size, loud)
    edge = 2 * size                                                # the last query opens a chunk: it sees itself alone
    chunk_case(path, dtype, H, G, d, dv, [edge + 1, 66], [edge, 65], size, edge - 1)


@pytest.mark.parametrize("d,splits", [(64, 1), (64, 4), (128, 3)])
def test_single_tokens_are_gated_in_the_attention_kernel(d, splits):
    o = ops()
    H, G, n = 6, 2, 3
    g = torch.Generator().manual_seed(d + splits)
    pasts = [200, 63, 0]
    k_pool, v_pool = (torch.randn(12, G, 64, d, generator=g).to(torch.bfloat16).to(DEV) for _ in range(2))
    table = i32([[3, 1, 7, 5], [0, 2, 4, 6], [8, 9, 10, 11]])
    q = torch.randn(n, H, d, generator=g).to(torch.bfloat16).to(DEV)
    _, _, start = batch_tables([1] * n, pasts)
    rows = torch.randn(n, H * d + 8, generator=g).to(DEV)
    outs = []
    for gate in (None, rows[:, 8:]):
        out = torch.empty(n, H * d, dtype=torch.bfloat16, device=DEV)
        scratch = torch.empty(max(o.decode_scratch_floats(n, H, d, splits), 1), device=DEV)
        o.attention_decode(q, k_pool, v_pool, out, start, i32(pasts), table, H, G, d, -100, 0.2, splits, scratch, sinks=torch.zeros(H, device=DEV), gate=gate)
        outs.append(out.float())
    torch.testing.assert_close(outs[1], outs[0] * torch.sigmoid(rows[:, 8:]), rtol=2e-2, atol=2e-3)


def test_the_one_in_the_denominator_counts_where_scores_are_low():
    """With every score far below zero almost nothing is attended to; a softmax without the one would return a mean."""
    o = ops()
    H, G, d, L = 2, 1, 64, 70
    for dtype in (torch.float32, torch.bfloat16):
        k_pool = torch.full((2, G, 64, d), -1.0, dtype=dtype, device=DEV)
        v_pool = torch.ones((2, G, 64, d), dtype=dtype, device=DEV)
        q = torch.ones(L, H, d, dtype=dtype, device=DEV)
        tok_seq, tok_pos, start = batch_tables([L])
        out = torch.empty(L, H * d, dtype=dtype, device=DEV)
        zeros = torch.zeros(H, device=DEV)
        table, scale = i32([[0, 1]]), 0.05
        if dtype == torch.float32:
            o.attention(q, k_pool, v_pool, out, tok_seq, tok_pos, table, H, G, d, 0, scale, sinks=zeros)
        else:
            o.attention_prefill(q, k_pool, v_pool, out, start, i32([0]), i32([L]), table, L, H, G, d, 0, scale, sinks=zeros)
        keys = torch.arange(1, L + 1, dtype=torch.float64)
        e = keys * torch.exp(torch.tensor(-64 * 0.05, dtype=torch.float64))
        torch.testing.assert_close(out[:, 0].cpu().double(), e / (1 + e), rtol=1e-2, atol=1e-3)


# ---------------------------------------------------------------- around the mixers ----

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,rot,tokens", [(4, 2, 24, 16, 16, 9), (6, 3, 64, 64, 64, 300), (8, 2, 64, 128, 32, 2), (3, 1, 18, 7, 0, 40), (5, 5, 128, 128, 128, 1100)])
def test_biases_and_whole_projection_norms_over_wider_rows(H, G, d, dv, rot, tokens, dtype):
    o = ops()
    g = torch.Generator().manual_seed(H * 31 + d)
    width = (H + G) * d + G * dv
    rows, bias = torch.randn(tokens, width + 8, generator=g), torch.randn(width, generator=g)
    qg, kg = torch.randn(H * d, generator=g) + 1, torch.randn(G * d, generator=g) + 1
    pages = (tokens + 63) // 64
    k_pool, v_pool = torch.zeros(pages, G, 64, d, dtype=dtype, device=DEV), torch.zeros(pages, G, 64, dv, dtype=dtype, device=DEV)
    tok_seq, tok_pos, _ = batch_tables([tokens])
    i = torch.arange(rot // 2, dtype=torch.float64)
    table = torch.arange(tokens, dtype=torch.float64)[:, None] * 100.0 ** (-2.0 * i / max(rot, 1))[None]
    q = torch.empty(tokens, H, d, dtype=dtype, device=DEV)
    o.qkv_post_span(rows.to(DEV)[:, :width], qg.to(DEV), kg.to(DEV), table.cos().float().to(DEV) if rot else None, table.sin().float().to(DEV) if rot else None,
                    q, k_pool, v_pool, tok_seq, tok_pos, i32([list(range(pages))]), H, G, d, dv, rot, True, True, 1e-5, bias=bias.to(DEV))
    r = rows[:, :width].double() + bias.double()
    ang = plain.angles(torch.arange(tokens), rot, 100.0, torch.float64)
    want_q = plain.rotate_neighbours((plain.rms(r[:, :H * d], 1e-5) * qg.double()).reshape(tokens, H, d), ang)
    want_k = plain.rotate_neighbours((plain.rms(r[:, H * d:(H + G) * d], 1e-5) * kg.double()).reshape(tokens, G, d), ang)
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    torch.testing.assert_close(q.cpu().double(), want_q, **tol)
    flat = lambda pool: pool.permute(0, 2, 1, 3).reshape(pages * 64, G, -1)[:tokens].cpu().double()
    torch.testing.assert_close(flat(k_pool), want_k, **tol)
    torch.testing.assert_close(flat(v_pool), r[:, (H + G) * d:].reshape(tokens, G, dv), **tol)


@pytest.mark.parametrize("d", [72, 256, 1024, 3000, 4100])
@pytest.mark.parametrize("pair", [False, True])
def test_the_closing_norm_joins_two_results_and_leaves_the_rounded_stream(d, pair):
    o = ops()
    g = torch.Generator().manual_seed(d)
    T, eps = 5, 1e-5
    x, y, y2 = (torch.randn(T, d, generator=g) for _ in range(3))
    w = torch.randn(d, generator=g) * 0.3
    dev, rounded = x.to(DEV), torch.empty(T, d, dtype=torch.bfloat16, device=DEV)
    o.gated_norm_add(dev, y.to(DEV), None, None, (1 + w).to(DEV), eps, second=(y2.to(DEV), 0.7, -1.3) if pair else None, rounded=rounded)
    joined = 0.7 * y.double() - 1.3 * y2.double() if pair else y.double()
    want = x.double() + plain.norm_about_one(joined, w.double(), eps)
    torch.testing.assert_close(dev.cpu().double(), want, rtol=1e-5, atol=1e-5)
    assert torch.equal(rounded, dev.to(torch.bfloat16))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("store", [False, True])
@pytest.mark.parametrize("E,same,top,d,ff,T", [(5, 2, 2, 40, 24, 3), (5, 2, 2, 72, 36, 90), (1, 3, 2, 48, 8, 50), (6, 2, 8, 64, 64, 150), (4, 4, 2, 256, 64, 700),
                                               (8, 8, 3, 64, 32, 7), (3, 0, 1, 40, 16, 33), (2, 2, 1, 66, 20, 65)])
def test_experts_that_return_their_input(E, same, top, d, ff, T, dtype, store):
    """Few pairs, tiles of pairs and (bfloat16, many pairs) the grouped tensor-memory products, with and without what was in
    the stream before."""
    o = ops()
    g = torch.Generator().manual_seed(E * 100 + T)
    w = {"router": torch.randn(E + same, d, generator=g) / d ** 0.5 * 2, "correction": torch.randn(E + same, generator=g) * 0.2}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"] = (torch.randn(ff, d, generator=g) / d ** 0.5 for _ in range(2))
        w[f"e{e}.down"] = torch.randn(d, ff, generator=g) / ff ** 0.5
    h, base = torch.randn(T, d, generator=g), torch.randn(T, d, generator=g)
    if dtype == torch.bfloat16:
        h = h.to(dtype).float()
        w = {k: v.to(dtype).float() if v.dim() > 1 and k != "router" else v for k, v in w.items()}
    m = {"router": {"experts": E, "identity": same, "top": top}}
    margins = []
    want = plain.experts(h.double(), {k: v.double() for k, v in w.items()}, "", m, margins)
    hd = h.to(dtype).to(DEV)
    gu = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(E)]).to(dtype).to(DEV)
    dn = torch.stack([w[f"e{e}.down"] for e in range(E)]).to(dtype).to(DEV)
    pairs = T * top
    choice, rank, place, order = (torch.zeros(pairs, dtype=torch.int32, device=DEV) for _ in range(4))
    counts = torch.zeros(E + same, dtype=torch.int32, device=DEV)
    weight, logits = torch.zeros(pairs, device=DEV), torch.zeros(T, E + same, device=DEV)
    grouped = dtype == torch.bfloat16 and pairs >= 1024
    tiles = torch.zeros(o.moe_tile_words(T, top, E + same), dtype=torch.int32, device=DEV) if grouped else None
    o.moe_route(hd, w["router"].to(DEV), None, choice, weight, rank, counts, place, order, top, None, logits, tiles, layout=pairs > o.MOE_FEW_PAIRS,
                scoring="softmax", pick_bias=w["correction"].to(DEV), identity=same)
    act = torch.full((pairs, ff), float("nan"), dtype=dtype, device=DEV)
    y = torch.full((pairs, d), float("nan"), device=DEV)
    x = torch.full((T, d), float("nan"), device=DEV) if store else base.to(DEV)
    if grouped:
        xs = torch.empty(pairs, d, dtype=dtype, device=DEV)
        o.moe_experts_tc(hd, gu, dn, order, place, weight, tiles, xs, act, y, x, top, choice=choice if same else None, store=store)
        o.gemm_tc_check(torch.device(DEV))
    else:
        o.moe_experts(hd, gu, dn, counts, order, weight, act, y, x, top, choice=choice, place=place, identity=same, store=store)
    clear = margins[0] > 1e-4
    assert int(clear.sum()) > 0.9 * T
    got = x.cpu().double() - (0 if store else base.double())
    tol = dict(rtol=2e-4, atol=2e-4) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)
    torch.testing.assert_close(got[clear], want[clear], **tol)
