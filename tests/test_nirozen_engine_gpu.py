"""The Nirozen model in the engine against the plain implementation, in float32 and bfloat16: whole prompts and the stream
after every layer run; prompts against token-by-token decoding; portions of several sizes down to two tokens; batches of
unequal requests against each alone, batch after batch through a cache with room for one (slots, pages and previous tokens
used again); the first tokens; long decoding across page borders; greedy generation through the entry point and its loop."""

from __future__ import annotations

import numpy as np
import pytest
import torch

import tiny_nirozen as tn
from closeness import check
from plain import nirozen_plain as plain
from plain.qwen3_plain import read_model

pytestmark = pytest.mark.gpu

# float32: the engine and the plain code differ by summation order only; every row is held to the bound. bfloat16: the plain
# code gets the weights rounded alike; activations and cache rows are rounded in the engine only, and where two router logits
# lie closer than that rounding the engine may send a token to another expert than the plain code does. Rows that such a
# close call can reach are left out (``Oracle.sure``).
TOL = {"fp32": dict(rtol=2e-4, atol=2e-4), "bf16": dict(rtol=0.0, atol=0.25)}
NAMES = ["S", "T", "U", "V", "W"]
LENGTHS = {"S": [1, 7, 66, 150], "T": [3, 64, 65, 200], "U": [2, 40, 129], "V": [5, 130, 300], "W": [1, 33, 260]}
CLEAR = 0.06        # a choice of experts is clear when the router logits at its edge differ by this much
COMPARED = {"fp32": 0, "bf16": 0}       # rows held to the plain implementation so far


def load(folder, dtype, max_tokens=2048, **kw):
    import sleuth_b200 as sb
    return sb.load(folder, dtype=dtype, max_seq_len=1024, max_tokens=max_tokens, **kw)


class Oracle:
    """The plain implementation's logits of a sequence, and which of its rows no close call among the experts can reach."""

    def __init__(self, folder, dtype):
        self.cfg, w = read_model(folder)
        if dtype == "bf16":
            # matrices are narrowed on the device; gains, biases, sinks, pass vectors and the routers' matrices stay float32
            w = {k: (v.to(torch.bfloat16).float() if v.is_floating_point() and v.dim() > 1 and not k.endswith((".router", "loop.step"))
                     else v) for k, v in w.items()}
        self.w, self.dtype, self.seen = w, dtype, {}
        self.last_is_own = self.cfg["layers"][plain.layer_runs(self.cfg)[-1][0]].get("mlp") is not None

    def _get(self, ids):
        key = tuple(ids)
        if key not in self.seen:
            margins = []
            logits = plain.forward(self.cfg, self.w, list(ids), torch.float64, margins=margins).float()
            sure = torch.ones(len(key), dtype=torch.bool)
            for n, m in enumerate(margins):
                clear = m > CLEAR
                # nothing attends after the last layer run: a close call there stays in its own row
                sure &= clear if self.last_is_own and n == len(margins) - 1 else clear.int().cumprod(0).bool()
            self.seen[key] = (logits, sure)
        return self.seen[key]

    def __call__(self, ids):
        return self._get(ids)[0]

    def sure(self, ids):
        return self._get(ids)[1] if self.dtype == "bf16" else torch.ones(len(ids), dtype=torch.bool)


def close(got, ref, ids, first=0):
    """``got``: the engine's logits of positions ``first`` ... of ``ids``."""
    got, want, sure = got.float().cpu(), ref(ids)[first:], ref.sure(ids)[first:]
    assert got.shape == want.shape and bool(torch.isfinite(got).all())
    COMPARED[ref.dtype] += int(sure.sum())
    if bool(sure.any()):
        check(got[sure], want[sure], TOL[ref.dtype], "nirozen " + ref.dtype)


def requests_for(name, lengths, seed=0, ref=None):
    """Random prompts; for a bfloat16 oracle, of up to 12 draws the one with the most rows out of reach of close calls."""
    rng = np.random.default_rng(seed + tn.SEEDS[name])
    out = []
    for n in lengths:
        draws = []
        for _ in range(12 if ref is not None and ref.dtype == "bf16" else 1):
            ids = rng.integers(0, tn.CONFIGS[name]["vocab"], size=n).tolist()
            draws.append((int(ref.sure(ids).sum()) if ref is not None else n, ids))
            if draws[-1][0] == n:
                break
        out.append(max(draws, key=lambda d: d[0])[1])
    return out


@pytest.fixture(scope="module")
def served(nirozen_folders):
    """Engines and oracles by (configuration, dtype), kept for the module."""
    kept = {}

    def get(name, dtype):
        if (name, dtype) not in kept:
            kept[name, dtype] = (load(nirozen_folders[name], dtype), Oracle(nirozen_folders[name], dtype))
        return kept[name, dtype]
    return get


both = pytest.mark.parametrize("dtype", ["fp32", "bf16"])
every = pytest.mark.parametrize("name", NAMES)


@both
@every
def test_whole_prompts_and_the_stream_after_every_layer(name, dtype, served):
    eng, ref = served(name, dtype)
    for ids in requests_for(name, LENGTHS[name], ref=ref):
        (slot,) = eng.open(1)
        got = eng.step([(slot, ids, tuple(range(len(ids))))])
        eng.close([slot])
        close(got, ref, ids)
    if dtype == "fp32":
        ids = requests_for(name, [21])[0]
        _, stream = plain.forward(ref.cfg, ref.w, ids, torch.float64, keep_stream=True)
        seen = []
        eng.model.observe = lambda i, x: seen.append(x.detach().cpu().clone())
        (slot,) = eng.open(1)
        eng.step([(slot, ids, (0,))])
        eng.close([slot])
        eng.model.observe = None
        assert len(seen) == stream.shape[0]
        for i, x in enumerate(seen):
            torch.testing.assert_close(x.double(), stream[i], rtol=1e-4, atol=1e-4 * float(stream[i].abs().max()))


@both
@every
def test_prompt_then_token_by_token(name, dtype, served):
    eng, ref = served(name, dtype)
    for ids in requests_for(name, [n for n in LENGTHS[name] if n > 40] + [34, 9], seed=1, ref=ref):
        cut = max(1, len(ids) - 33)
        (slot,) = eng.open(1)
        rows = [eng.step([(slot, ids[:cut], (cut - 1,))]).cpu()]
        rows += [eng.step([(slot, [t], (0,))]).cpu().clone() for t in ids[cut:]]
        eng.close([slot])
        close(torch.cat(rows), ref, ids, cut - 1)


@both
@every
def test_from_the_first_token_on_one_by_one(name, dtype, served):
    eng, ref = served(name, dtype)
    ids = requests_for(name, [70], seed=2, ref=ref)[0]
    (slot,) = eng.open(1)
    rows = [eng.step([(slot, [t], (0,))]).cpu().clone() for t in ids]
    eng.close([slot])
    close(torch.cat(rows), ref, ids)


@both
@every
@pytest.mark.parametrize("portion", [2, 7, 64, 100])
def test_portions_of_a_prompt(name, portion, dtype, served, nirozen_folders):
    eng, ref = served(name, dtype)
    ids = requests_for(name, [131], seed=3, ref=ref)[0]
    (slot,) = eng.open(1)
    rows = []
    for a in range(0, len(ids), portion):
        part = ids[a:a + portion]
        rows.append(eng.step([(slot, part, tuple(range(len(part))))]).cpu().clone())
    eng.close([slot])
    close(torch.cat(rows), ref, ids)
    if dtype == "fp32":         # and through the stepper's own cutting of long steps
        small = load(nirozen_folders[name], dtype, max_step_tokens=portion + 1)
        (slot,) = small.open(1)
        close(small.step([(slot, ids, tuple(range(len(ids))))]), ref, ids)


@both
@pytest.mark.parametrize("name", ["V", "T"])
def test_a_long_prompt_in_two_large_portions(name, dtype, served):
    """The first portion may run on per-head keys and values, the second reads what it left in the cache."""
    eng, ref = served(name, dtype)
    ids = requests_for(name, [400], seed=7, ref=ref)[0]
    (slot,) = eng.open(1)
    rows = [eng.step([(slot, part, tuple(range(len(part))))]).cpu().clone() for part in (ids[:250], ids[250:])]
    eng.close([slot])
    close(torch.cat(rows), ref, ids)


@both
@every
def test_unequal_batches_one_after_another_reuse_slots_and_pages(name, dtype, nirozen_folders, served):
    """Three batches through a cache with room for one. Prompts and numbers of decoded tokens are unequal, the shorter
    requests end earlier, and the next batch gets slots and pages still full of the last one's rows."""
    eng, ref = load(nirozen_folders[name], dtype, max_tokens=64 * 8), served(name, dtype)[1]
    plans = [[(100, 20), (60, 3), (5, 27)], [(1, 12), (64, 1), (63, 2), (30, 30)], [(190, 9), (2, 40), (129, 2)]]
    for b, plan in enumerate(plans):
        reqs = requests_for(name, [p + d for p, d in plan], seed=10 + b, ref=ref)
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
            close(torch.stack(got[i]), ref, ids, p - 1)
        assert eng.cache.book.pages_in_use() == [0] * eng.cache.n_groups


@both
def test_a_mixed_step_of_portions_and_single_tokens(dtype, served):
    """Sequences that go on by one token, by a few and by many, and one that starts, in the same step."""
    eng, ref = served("V", dtype)
    reqs = requests_for("V", [140, 90, 70, 131], seed=8, ref=ref)
    held = [139, 80, 5, 0]
    slots = eng.open(4)
    eng.step([(s, ids[:n], ()) for s, ids, n in zip(slots[:3], reqs, held)])
    out = eng.step([(s, ids[n:], tuple(range(len(ids) - n))) for s, ids, n in zip(slots, reqs, held)]).cpu()
    eng.close(slots)
    at = 0
    for ids, n in zip(reqs, held):
        close(out[at:at + len(ids) - n], ref, ids, n)
        at += len(ids) - n


@both
def test_a_slot_taken_again_starts_from_nothing(dtype, nirozen_folders, served):
    """One slot, one request after another: the previous token of the request before must not reach the next one, whose
    first token is a sequence's first token again."""
    eng, ref = load(nirozen_folders["S"], dtype, max_tokens=128, max_sequences=1), served("S", dtype)[1]
    for ids in requests_for("S", [50, 1, 33, 2], seed=8, ref=ref):
        (slot,) = eng.open(1)
        assert slot == 0
        rows = [eng.step([(slot, ids[:1], (0,))]).cpu().clone()]
        if len(ids) > 1:
            rows.append(eng.step([(slot, ids[1:], tuple(range(len(ids) - 1)))]).cpu().clone())
        eng.close([slot])
        close(torch.cat(rows), ref, ids)


@both
@pytest.mark.parametrize("name", ["S", "V"])
def test_long_decoding_across_page_borders(name, dtype, served):
    eng, ref = served(name, dtype)
    ids = requests_for(name, [330], seed=4, ref=ref)[0]
    (slot,) = eng.open(1)
    rows = [eng.step([(slot, ids[:60], (59,))]).cpu()]
    rows += [eng.step([(slot, [t], (0,))]).cpu().clone() for t in ids[60:]]
    eng.close([slot])
    close(torch.cat(rows), ref, ids, 59)


def test_float32_does_not_depend_on_the_batch(served):
    eng, _ = served("T", "fp32")
    reqs = requests_for("T", [90, 3, 41], seed=5)
    alone = []
    for ids in reqs:
        (slot,) = eng.open(1)
        alone.append(eng.step([(slot, ids, (len(ids) - 1,))]).cpu().clone())
        eng.close([slot])
    slots = eng.open(3)
    together = eng.step([(s, ids, (len(ids) - 1,)) for s, ids in zip(slots, reqs)]).cpu()
    eng.close(slots)
    torch.testing.assert_close(together, torch.cat(alone), rtol=1e-5, atol=1e-5)


@both
@pytest.mark.parametrize("name", ["S", "V"])
def test_greedy_generation_through_the_entry_point(name, dtype, served):
    """Unequal prompts through ``Engine.generate`` (its loop, its device-fed decode steps, its sampler) against greedy
    decoding with the plain implementation, which follows the engine's tokens: at every step the engine's token must be
    the plain code's best, or, where its two best logits lie closer than the run's rounding, one of those two."""
    import sleuth_b200 as sb
    eng, ref = served(name, dtype)
    prompts = requests_for(name, [3, 70, 20, 1, 9, 130], seed=6, ref=ref)
    out = eng.generate(prompts, max_new_tokens=12, sampling=sb.SamplingConfig(temperature=0), stop_ids=())
    margin = {"fp32": 1e-3, "bf16": 0.25}[dtype]
    clear = checked = 0
    for ids, r in zip(prompts, out):
        assert len(r.new_ids) == 12
        seq = list(ids)
        for tok in r.new_ids:
            if bool(ref.sure(seq)[-1]):
                top2 = torch.topk(ref(seq)[-1], 2)
                if float(top2.values[0] - top2.values[1]) >= margin:
                    assert tok == int(top2.indices[0])
                    clear += 1
                else:
                    assert tok in top2.indices.tolist()
                checked += 1
            seq.append(tok)
    assert checked >= {"fp32": 72, "bf16": 6}[dtype] and (dtype == "bf16" or clear >= 50)


def test_zz_enough_bfloat16_rows_were_held_to_the_plain_implementation():
    """The bfloat16 comparisons leave out rows that a close call can reach; this many were compared all the same (run
    after the tests above)."""
    if COMPARED["fp32"] > 3000:          # the whole file ran
        assert COMPARED["bf16"] > 2000, COMPARED
