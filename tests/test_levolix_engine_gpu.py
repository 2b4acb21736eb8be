"""The Levolix model in the engine against the plain implementation, in float32 and bfloat16: whole prompts and the stream
after every layer; prompts against token-by-token decoding; portions of several sizes down to two tokens; batches of unequal
requests against each alone, batch after batch through a cache with room for one (slots, pages, states and convolution tails
used again); the first tokens; long decoding across page and chunk borders; greedy generation through the entry point and its
loop."""

from __future__ import annotations

import numpy as np
import pytest
import torch

import tiny_levolix as tl
from closeness import check
from plain import levolix_plain as plain
from plain.qwen3_plain import read_model

pytestmark = pytest.mark.gpu

# float32: the engine and the plain code differ by summation order only. bfloat16: weights are compared rounded alike;
# activations and cache rows are rounded in the engine only. A rounding that turns one choice of experts changes everything
# behind it, so bfloat16 runs use the folders whose choices the corrections alone make (the weights stay the token's scores).
# Where a head's result is small beside the terms it sums (q . k near zero at a first token, say), its norm magnifies their rounding: one row in forty (or one) may
# exceed the bfloat16 bound, which is about ten times the median of the rows' largest differences (logits go up to 29).
TOL = {"fp32": dict(rtol=3e-4, atol=3e-3), "bf16": dict(rtol=0.0, atol=1.2)}
NAMES = ["F", "H", "J"]
LENGTHS = {"F": [1, 7, 66, 150], "H": [3, 64, 65, 210], "J": [2, 40, 129]}


def folder_of(folders, name, dtype):
    return folders[name + " steady" if dtype == "bf16" else name]


def load(folder, dtype, max_tokens=2048, **kw):
    import sleuth_b200 as sb
    return sb.load(folder, dtype=dtype, max_seq_len=1024, max_tokens=max_tokens, **kw)


def oracle(folder, dtype):
    cfg, w = read_model(folder)
    if dtype == "bf16":     # matrices are narrowed on the device; gains, biases, taps and the routers' matrices stay float32
        w = {k: (v.to(torch.bfloat16).float() if v.is_floating_point() and v.dim() > 1 and not k.endswith((".router", ".conv")) else v)
             for k, v in w.items()}
    cache, streams = {}, {}

    def f(ids):
        key = tuple(ids)
        if key not in cache:
            logits, streams[key] = plain.forward(cfg, w, torch.tensor(list(ids)), torch.float64)
            cache[key] = logits.float()
        return cache[key]

    def stream(ids):
        f(ids)
        return streams[tuple(ids)]
    f.stream = stream
    return f


def close(got, want, dtype, label):
    got, want = got.float().cpu(), want.float().cpu()
    assert bool(torch.isfinite(got).all()) and got.shape == want.shape
    if dtype == "bf16":
        over = (got - want).abs().amax(dim=-1) > TOL[dtype]["atol"]
        assert int(over.sum()) <= max(1, len(over) // 40), (got - want).abs().amax(dim=-1)
        got, want = got[~over], want[~over]
    check(got, want, TOL[dtype], label)


def requests_for(name, lengths, seed=0):
    rng = np.random.default_rng(seed + tl.SEEDS[name])
    return [rng.integers(0, tl.CONFIGS[name]["vocab"], size=n).tolist() for n in lengths]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(name, dtype, levolix_folders):
    eng, ref = load(folder_of(levolix_folders, name, dtype), dtype), oracle(folder_of(levolix_folders, name, dtype), dtype)
    for ids in requests_for(name, LENGTHS[name]):
        (slot,) = eng.open(1)
        got = eng.step([(slot, ids, tuple(range(len(ids))))]).cpu()
        eng.close([slot])
        close(got, ref(ids), dtype, "levolix " + dtype)


@pytest.mark.parametrize("name", NAMES)
def test_the_stream_after_every_layer(name, levolix_folders):
    eng, ref = load(levolix_folders[name], "fp32"), oracle(levolix_folders[name], "fp32")
    ids = requests_for(name, [21])[0]
    seen = []
    eng.model.observe = lambda i, x: seen.append(x.detach().cpu().clone())
    (slot,) = eng.open(1)
    eng.step([(slot, ids, (0,))])
    eng.close([slot])
    eng.model.observe = None
    want = ref.stream(ids)
    assert len(seen) == want.shape[0]
    for i, x in enumerate(seen):
        torch.testing.assert_close(x.double(), want[i], rtol=1e-4, atol=1e-4 * float(want[i].abs().max()))


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_token_by_token(name, dtype, levolix_folders):
    eng, ref = load(folder_of(levolix_folders, name, dtype), dtype), oracle(folder_of(levolix_folders, name, dtype), dtype)
    for ids in requests_for(name, [n for n in LENGTHS[name] if n > 40] + [34, 9], seed=1):
        cut = max(1, len(ids) - 33)
        (slot,) = eng.open(1)
        rows = [eng.step([(slot, ids[:cut], (cut - 1,))]).cpu()]
        for t in ids[cut:]:
            rows.append(eng.step([(slot, [t], (0,))]).cpu().clone())
        eng.close([slot])
        close(torch.cat(rows), ref(ids)[cut - 1:], dtype, "levolix " + dtype)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", NAMES)
def test_from_the_first_token_on_one_by_one(name, dtype, levolix_folders):
    eng, ref = load(folder_of(levolix_folders, name, dtype), dtype), oracle(folder_of(levolix_folders, name, dtype), dtype)
    ids = requests_for(name, [70], seed=2)[0]
    (slot,) = eng.open(1)
    rows = [eng.step([(slot, [t], (0,))]).cpu().clone() for t in ids]
    eng.close([slot])
    close(torch.cat(rows), ref(ids), dtype, "levolix " + dtype)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("portion", [2, 3, 64, 100])
def test_portions_of_a_prompt(name, portion, dtype, levolix_folders):
    """Portions shorter than a convolution (its tail then mixes old and new inputs), of a page, and longer."""
    eng, ref = load(folder_of(levolix_folders, name, dtype), dtype), oracle(folder_of(levolix_folders, name, dtype), dtype)
    ids = requests_for(name, [131], seed=3)[0]
    (slot,) = eng.open(1)
    rows = []
    for a in range(0, len(ids), portion):
        part = ids[a:a + portion]
        rows.append(eng.step([(slot, part, tuple(range(len(part))))]).cpu().clone())
    eng.close([slot])
    close(torch.cat(rows), ref(ids), dtype, "levolix " + dtype)
    if dtype == "fp32":         # and through the stepper's own cutting of long steps
        small = load(folder_of(levolix_folders, name, dtype), dtype, max_step_tokens=portion + 1)
        (slot,) = small.open(1)
        got = small.step([(slot, ids, tuple(range(len(ids))))]).cpu()
        close(got, ref(ids), dtype, "levolix " + dtype)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_one_after_another_reuse_slots_and_pages(name, dtype, levolix_folders):
    """Three batches through a cache with room for one. Prompts and numbers of decoded tokens are unequal, the shorter
    requests end earlier, and the next batch gets slots, pages, states and tails still full of the last one's."""
    eng, ref = load(folder_of(levolix_folders, name, dtype), dtype, max_tokens=64 * 8), oracle(folder_of(levolix_folders, name, dtype), dtype)
    plans = [[(100, 20), (60, 3), (5, 27)], [(1, 12), (64, 1), (63, 2), (30, 30)], [(190, 9), (2, 40)]]
    for b, plan in enumerate(plans):
        reqs = requests_for(name, [p + d for p, d in plan], seed=10 + b)
        slots = eng.open(len(reqs))
        got = {i: [] for i in range(len(reqs))}
        out = eng.step([(s, ids[:p], (p - 1,)) for s, ids, (p, d) in zip(slots, reqs, plan)]).cpu()
        for i in range(len(reqs)):
            got[i].append(out[i])
        live, k = list(range(len(reqs))), 0
        while live:
            out = eng.step([(slots[i], [reqs[i][plan[i][0] + k]], (0,)) for i in live]).cpu()
            for j, i in enumerate(live):
                got[i].append(out[j].clone())
            k += 1
            done = [i for i in live if k >= plan[i][1]]
            eng.close([slots[i] for i in done])
            live = [i for i in live if i not in done]
        for i, (ids, (p, d)) in enumerate(zip(reqs, plan)):
            close(torch.stack(got[i]), ref(ids)[p - 1:], dtype, "levolix " + dtype)
        assert eng.cache.book.pages_in_use() == [0] * eng.cache.n_groups


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_a_slot_taken_again_starts_from_nothing(dtype, levolix_folders):
    """One slot, one request after another: the states and convolution tails of the request before must not reach the
    next one, whose first tokens see zeros in front of them again."""
    eng, ref = load(folder_of(levolix_folders, "F", dtype), dtype, max_tokens=128, max_sequences=1), oracle(folder_of(levolix_folders, "F", dtype), dtype)
    for ids in requests_for("F", [50, 1, 33, 2], seed=8):
        (slot,) = eng.open(1)
        assert slot == 0
        rows = [eng.step([(slot, ids[:1], (0,))]).cpu().clone()]
        if len(ids) > 1:
            rows.append(eng.step([(slot, ids[1:], tuple(range(len(ids) - 1)))]).cpu().clone())
        eng.close([slot])
        close(torch.cat(rows), ref(ids), dtype, "levolix " + dtype)


def test_the_cache_of_a_chunked_layer_gives_pages_back(levolix_folders):
    eng = load(levolix_folders["F"], "fp32", max_tokens=64 * 12)
    ids = requests_for("F", [600], seed=9)[0]
    (slot,) = eng.open(1)
    eng.step([(slot, ids[:500], ())])
    for t in ids[500:]:
        eng.step([(slot, [t], ())])
    windows = [g.window for g in eng.cache.book.groups]
    used = eng.cache.book.pages_in_use()
    assert sorted(windows) == [-64, -37]
    # 600 = 9 * 64 + 24 = 16 * 37 + 8: the next token sees positions 576 .. of the chunks of 64, 592 .. of those of 37
    assert used[windows.index(-64)] == 1 and used[windows.index(-37)] == 1
    eng.close([slot])


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", ["F", "H"])
def test_long_decoding_across_page_and_chunk_borders(name, dtype, levolix_folders):
    eng, ref = load(folder_of(levolix_folders, name, dtype), dtype), oracle(folder_of(levolix_folders, name, dtype), dtype)
    ids = requests_for(name, [330], seed=4)[0]
    (slot,) = eng.open(1)
    rows = [eng.step([(slot, ids[:60], (59,))]).cpu()]
    for t in ids[60:]:
        rows.append(eng.step([(slot, [t], (0,))]).cpu().clone())
    close(torch.cat(rows), ref(ids)[59:], dtype, "levolix " + dtype)


def test_float32_does_not_depend_on_the_batch(levolix_folders):
    eng = load(levolix_folders["H"], "fp32")
    reqs = requests_for("H", [90, 3, 41], seed=5)
    alone = []
    for ids in reqs:
        (slot,) = eng.open(1)
        alone.append(eng.step([(slot, ids, (len(ids) - 1,))]).cpu().clone())
        eng.close([slot])
    slots = eng.open(3)
    together = eng.step([(s, ids, (len(ids) - 1,)) for s, ids in zip(slots, reqs)]).cpu()
    torch.testing.assert_close(together, torch.cat(alone), rtol=1e-4, atol=1e-3)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", ["F", "H"])
def test_greedy_generation_through_the_entry_point(name, dtype, levolix_folders):
    """Unequal prompts through ``Engine.generate`` (its loop, its device-fed decode steps, its sampler) against greedy
    decoding with the plain implementation, which follows the engine's tokens."""
    import sleuth_b200 as sb
    eng, ref = load(folder_of(levolix_folders, name, dtype), dtype), oracle(folder_of(levolix_folders, name, dtype), dtype)
    prompts = requests_for(name, [3, 70, 20, 1, 9, 130], seed=6)
    out = eng.generate(prompts, max_new_tokens=12, sampling=sb.SamplingConfig(temperature=0), stop_ids=())
    margin = {"fp32": 1e-3, "bf16": TOL["bf16"]["atol"]}[dtype]      # the engine's token is the plain code's best, or within the run's rounding of it
    clear = near = checked = 0
    for ids, r in zip(prompts, out):
        assert len(r.new_ids) == 12
        seq = list(ids)
        for tok in r.new_ids:
            row = ref(seq)[-1]
            near += int(float(row.max() - row[tok]) <= margin)
            clear += int(tok == int(row.argmax()))
            checked += 1
            seq.append(tok)
    assert checked == near == 72 and clear >= checked * 0.7
