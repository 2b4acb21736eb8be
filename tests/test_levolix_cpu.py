"""Levolix without a GPU: the configuration reader (nested keys, refusals), the model description (tensor names and shapes, cache
requests, layers without front norms), the book of a chunked layer, and identities of the plain implementation itself (a
recurrence or a convolution cut anywhere, the delta rule's replacement of a value, chunk membership, the one in the softmax
denominator, both rotations, identity experts)."""

from __future__ import annotations

import copy

import pytest
import torch

import tiny_levolix as tl
from plain import levolix_plain as plain
from sleuth_b200.config import ConfigError, parse_config
from sleuth_b200.engine.model import declare_model


def spec_of(cfg):
    arch, c, unread = parse_config(cfg)
    assert arch.name == "Levolix" and not unread
    return arch.model_spec(c)


@pytest.mark.parametrize("name", list(tl.CONFIGS))
def test_the_description_names_every_tensor_once(name):
    cfg = tl.CONFIGS[name]
    decl = declare_model(spec_of(cfg))
    d, seen = cfg["width"], {"embed", "final.norm"}
    assert decl["embed"].shape == (cfg["vocab"], d) and decl["final.norm"].shape == (d,)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        want = {"norm1": (d,)}
        if L["type"] == "retention":
            nk, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            want.update({"mix.q": (nk, d), "mix.k": (nk, d), "mix.v": (nv, d), "mix.g": (nv, d), "mix.o": (d, nv)})
        else:
            a, r = m["left"], m["right"]
            nq, nk, nv, no = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"], a["heads"] * a["vdim"]
            for n, rows in (("q", nq), ("k", nk), ("v", nv)):
                want[f"mix.left.{n}"], want[f"mix.left.{n}.b"] = (rows, d), (rows,)
            want.update({"mix.left.q.norm": (nq,), "mix.left.k.norm": (nk,), "mix.left.g": (no, d), "mix.left.o": (d, no)})
            nk, nv, H = r["kv_heads"] * r["dim"], r["heads"] * r["vdim"], r["heads"]
            for n, rows in (("q", nk), ("k", nk), ("v", nv)):
                want[f"mix.right.{n}"], want[f"mix.right.{n}.conv"] = (rows, d), (rows, r["conv"])
            want.update({"mix.right.b": (H, d), "mix.right.a": (H, d), "mix.right.A_log": (H,), "mix.right.dt_bias": (H,), "mix.right.norm": (r["vdim"],),
                         "mix.right.g": (nv, d), "mix.right.o": (d, nv)})
        if L["mlp"]:
            ro, ff = L["mlp"]["router"], L["mlp"]["expert"]["ff"]
            want.update({"norm2": (d,), "mlp.router": (ro["experts"] + ro["identity"], d), "mlp.correction": (ro["experts"] + ro["identity"],)})
            for e in range(ro["experts"]):
                want.update({f"mlp.e{e}.gate": (ff, d), f"mlp.e{e}.up": (ff, d), f"mlp.e{e}.down": (d, ff)})
        for n, shape in want.items():
            assert tuple(decl[p + n].shape) == shape, p + n
            seen.add(p + n)
    assert set(decl) == seen


def test_cache_requests_bundle_pages_states_and_tails():
    from sleuth_b200.cache.paged import KVRequest, StateRequest, leaf_requests
    from sleuth_b200.engine.model import Model
    from sleuth_b200.parts.base import BuildContext
    model = Model(spec_of(tl.F), BuildContext(device=torch.device("cpu"), dtype=torch.float32, max_positions=64))
    leaves = [list(leaf_requests(r)) for r in model.cache_requests]
    assert leaves[0] == [StateRequest((3, 12, 20))] and leaves[2] == [StateRequest((1, 40, 72))]
    assert leaves[1] == [KVRequest(2, 24, -37, 16), StateRequest((6, 12, 10)), StateRequest((2, 2 * 2 * 12 + 6 * 10))]
    assert leaves[3] == [KVRequest(3, 16, -64, 40), StateRequest((2, 40, 24))]           # one tap: no tail
    assert model.reads_stream and model.layers[0].norm1 is None


def test_refusals():
    def broken(change):
        cfg = copy.deepcopy(tl.F)
        change(cfg)
        with pytest.raises(ConfigError):
            spec_of(cfg)
    left, right = (lambda c: c["layers"][1]["mixer"]["left"]), (lambda c: c["layers"][1]["mixer"]["right"])
    broken(lambda c: c["layers"][0].update(type="serial"))
    broken(lambda c: left(c).update(heads=3))                                       # 3 query heads on 2 key/value heads
    broken(lambda c: left(c).update(window=5))                                      # an unknown key
    broken(lambda c: left(c)["mask"].update(size=0))
    broken(lambda c: left(c)["rot"].update(dims=26))                                # more than the head has
    broken(lambda c: right(c).update(kv_heads=4))
    broken(lambda c: right(c).update(conv=0))
    broken(lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.5]))              # two decays for three heads
    broken(lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.5, -0.1]))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=8))                 # of 5 + 2
    broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda c: c["layers"][1]["mixer"].pop("left_scale"))


def test_the_book_of_a_chunked_group():
    from sleuth_b200.cache.book import CacheBook, first_visible
    assert [first_visible(p, -37) for p in (0, 36, 37, 73, 74)] == [0, 0, 37, 37, 74]
    assert [first_visible(p, 3) for p in (0, 2, 3, 9)] == [0, 0, 1, 7] and first_visible(9, 0) == 0
    for size in (1, 37, 64, 100, 128, 4000):
        book = CacheBook([-size, 0], 40, 2, 32)
        (s,) = book.open(1)
        n = 0
        for take in [100, 1, 1, 27, 64, 63, *[1] * 140]:
            n += take
            book.grow([s], [n])
            held = {i for i, p in enumerate(book.groups[0].table[s]) if p >= 0}
            assert set(range((n - take) // size * size // 64, (n - 1) // 64 + 1)) <= held       # what the step's queries read and write
            book.commit([s], [n])
            held = {i for i, p in enumerate(book.groups[0].table[s]) if p >= 0}
            assert held == set(range(n // size * size // 64, (n - 1) // 64 + 1))                # and nothing that no later query sees
        book.close([s])
        assert book.pages_in_use() == [0, 0]


def test_recurrences_cut_anywhere_with_their_state():
    g = torch.Generator().manual_seed(1)
    T, H, N, P = 30, 2, 5, 3
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    k, q, v, beta, dec = plain.unit(rnd(T, H, N)), rnd(T, H, N), rnd(T, H, P), torch.sigmoid(rnd(T, H)), torch.sigmoid(rnd(T, H))
    fixed = torch.tensor([0.9, 0.5], dtype=torch.float64)
    whole, last = plain.delta_recurrence(dec, beta, k, v, q)
    whole_f, last_f = plain.decayed_recurrence(fixed, k, v, q)
    for cut in (1, 7, 29):
        _, S = plain.delta_recurrence(dec[:cut], beta[:cut], k[:cut], v[:cut], q[:cut])
        rest, S2 = plain.delta_recurrence(dec[cut:], beta[cut:], k[cut:], v[cut:], q[cut:], S)
        torch.testing.assert_close(rest, whole[cut:])
        torch.testing.assert_close(S2, last)
        _, S = plain.decayed_recurrence(fixed, k[:cut], v[:cut], q[:cut])
        rest, S2 = plain.decayed_recurrence(fixed, k[cut:], v[cut:], q[cut:], S)
        torch.testing.assert_close(rest, whole_f[cut:])
        torch.testing.assert_close(S2, last_f)


def test_the_delta_rule_replaces_what_a_key_holds():
    key = torch.tensor([[[0.6, 0.8]]], dtype=torch.float64)
    one = torch.ones(1, 1, dtype=torch.float64)
    _, S = plain.delta_recurrence(one, one, key, torch.tensor([[[5.0, -1.0]]], dtype=torch.float64), key)
    out, S = plain.delta_recurrence(one, one, key, torch.tensor([[[2.0, 7.0]]], dtype=torch.float64), key, S)
    torch.testing.assert_close(out[0, 0], torch.tensor([2.0, 7.0], dtype=torch.float64))       # and the read-out sees the write


def test_chunk_membership_and_the_one_in_the_denominator():
    seen = plain.same_chunk(10, 3)
    assert seen[5].nonzero().flatten().tolist() == [3, 4, 5] and seen[6].nonzero().flatten().tolist() == [6]
    assert plain.same_chunk(4, 100).tril().sum() == 10 and plain.same_chunk(4, 1).sum() == 4
    s = torch.tensor([[1.0, -2.0, 300.0], [-300.0, -400.0, 0.0]], dtype=torch.float64)
    p = plain.softmax_plus_one(s, torch.tensor([[True, True, False], [True, True, False]]))
    e = torch.exp(s[0, :2])
    torch.testing.assert_close(p[0, :2], e / (1 + e.sum()))
    assert float(p[0, 2]) == 0 and float(p[1].sum()) < 1e-100


def test_both_rotations_turn_pairs_by_the_same_angles():
    g = torch.Generator().manual_seed(2)
    v, ang = torch.randn(7, 2, 12, generator=g, dtype=torch.float64), plain.angles(torch.arange(7), 8, 100.0, torch.float64)
    order = [0, 4, 1, 5, 2, 6, 3, 7, 8, 9, 10, 11]              # halves laid out as neighbours
    torch.testing.assert_close(plain.rotate_halves(v, ang)[..., order], plain.rotate_neighbours(v[..., order], ang))
    assert torch.equal(plain.rotate_halves(v, ang)[..., 8:], v[..., 8:]) and torch.equal(plain.rotate_neighbours(v, ang)[0], v[0])


def test_identity_experts_weigh_the_input_and_the_correction_moves_the_choice_only():
    g = torch.Generator().manual_seed(3)
    d, E = 12, 3
    w = {"router": torch.randn(E + 2, d, generator=g).double(), "correction": torch.zeros(E + 2, dtype=torch.float64)}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = (torch.randn(s, generator=g).double() for s in ((4, d), (4, d), (d, 4)))
    h = torch.randn(6, d, generator=g).double()
    s = torch.softmax(h @ w["router"].T, dim=-1)
    every = sum(s[:, e:e + 1] * plain.expert(h, w, f"e{e}.") for e in range(E)) + (s[:, 3:4] + s[:, 4:5]) * h
    torch.testing.assert_close(plain.experts(h, w, "", {"router": {"experts": E, "identity": 2, "top": 5}}), every)
    w["correction"][4] = 10.0
    torch.testing.assert_close(plain.experts(h, w, "", {"router": {"experts": E, "identity": 2, "top": 1}}), s[:, 4:5] * h)
