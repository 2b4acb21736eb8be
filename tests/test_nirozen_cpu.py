"""Nirozen without a GPU: its configuration, its model description, its tensors, refusals, and the plain implementation's own
consistency (the sink as one more key without value, the position vector, gains stored less one, the pair table's rows, the
carried form of latent attention, the order of layer runs)."""

from __future__ import annotations

import copy
import math

import pytest
import torch

import tiny_nirozen as tn
from plain import nirozen_plain as plain
from plain.qwen3_plain import read_model
from sleuth_b200.config import ConfigError, parse_config
from sleuth_b200.engine.model import declare_model
from sleuth_b200.parts.base import BuildContext, build_norm
from sleuth_b200.parts.ends import sinusoid_turns
from sleuth_b200.parts.spec import NormSpec, looped_schedule


def spec_of(cfg):
    arch, typed, unread = parse_config(cfg)
    assert arch.name == "Nirozen" and set(unread) <= {"torch_dtype"}      # the folder writer's own note
    return arch.model_spec(typed)


def test_every_size_and_constant_comes_from_the_configuration():
    spec = spec_of(tn.S)
    m = spec.layers[0].mixer
    assert (m.heads, m.plain_dim, m.rot_dim, m.value_dim, m.q_rank, m.kv_rank, m.window) == (3, 12, 0, 20, 28, 36, 0)
    assert m.scale == 0.37 and m.norm_eps == 1e-6 and m.sinks and m.output_gate and m.gate_span == "channel"
    assert m.position.kind == "none"
    assert (spec.layers[1].mixer.heads, spec.layers[1].mixer.q_rank, spec.layers[2].mixer.kv_rank) == (5, 50, 44)
    e = spec.embedding
    assert (e.kind, e.vocab, e.dim, e.buckets, e.mul_prev, e.mul_cur, e.scale) == ("pair_embedding", 211, 75, 89, 7, 13, 11.0)
    assert e.sinusoid == 10000.0
    assert spec.head.norm.gain_offset == 1.0 and spec.head.norm.eps == 1e-6 and not spec.head.tied
    f = spec.layers[0].ffn
    assert (f.experts, f.top, f.intermediate, f.scoring, f.router_bias, f.choice_bias) == (5, 2, 18, "softmax_top", True, False)
    assert f.activation == "silu" and f.shared.intermediate == 26 and f.shared.activation == "silu"
    assert spec.layers[1].ffn is None and spec.layers[1].norm2 is None and spec.layers[2].ffn.shared.intermediate == 10
    assert all(L.kind == "prenorm" and L.norm1.gain_offset == 1.0 and L.norm1.eps == 1e-6 for L in spec.layers)
    t = spec_of(tn.T)
    assert t.layers[1].ffn.shared is None and t.layers[1].mixer.scale == 0.2 and t.layers[0].norm1.eps == 2e-5
    bare = copy.deepcopy(tn.S)
    bare["embedding"] = {"scale": 2.0}
    assert spec_of(bare).embedding.kind == "token_embedding" and spec_of(bare).embedding.sinusoid == 10000.0


def test_the_loop_becomes_a_schedule_with_caches_of_its_own():
    spec = spec_of(tn.S)
    assert [(e.layer, e.add_row) for e in spec.schedule] == [(0, -1), (1, 0), (2, -1), (1, 1), (2, -1)]
    assert [e.cache for e in spec.schedule] == list(range(5)) and spec.pass_rows == "loop.step" and spec.pass_rows_count == 2
    assert not any(e.add_embedding or e.mix_embedding for e in spec.schedule) and spec.pass_mix is None
    assert [(e.layer, e.add_row) for e in spec_of(tn.T).schedule] == [(0, 0), (1, -1), (0, 1), (1, -1), (0, 2), (1, -1)]
    none = spec_of(tn.U)
    assert none.pass_rows is None and len(none.schedule) == 3 and none.ignored_tensors
    assert [(e.layer, e.add_row) for e in spec_of(tn.V).schedule] == [(0, -1), (1, -1), (2, 0)]
    assert plain.layer_runs(tn.S) == [(0, None), (1, 0), (2, None), (1, 1), (2, None)]
    with pytest.raises(ValueError):
        looped_schedule(3, 0, 2, 2, entry="rows")


def test_declared_tensors_carry_the_file_names_and_shapes():
    d = declare_model(spec_of(tn.S))
    assert d["embed"].shape == (211, 75) and d["bigram"].shape == (90, 75) and d["head"].shape == (211, 75)
    assert d["final.norm"].shape == (75,) and d["final.norm"].role == "vector" and d["loop.step"].shape == (2, 75)
    assert d["l0.mix.dq"].shape == (28, 75) and d["l0.mix.dq.norm"].shape == (28,) and d["l0.mix.uq"].shape == (36, 28)
    assert d["l0.mix.dkv"].shape == (36, 75) and d["l0.mix.dkv.norm"].shape == (36,)
    assert d["l0.mix.uk"].shape == (36, 36) and d["l0.mix.uv"].shape == (60, 36)
    assert d["l0.mix.sink"].shape == (3,) and d["l0.mix.sink"].role == "vector"
    assert d["l0.mix.g"].shape == (60, 75) and d["l0.mix.o"].shape == (75, 60)
    assert d["l0.mlp.router"].shape == (5, 75) and d["l0.mlp.router.b"].shape == (5,)
    assert d["l0.mlp.e4.up"].shape == (18, 75) and d["l0.mlp.shared.down"].shape == (75, 26)
    assert "l1.norm2" not in d and "l1.mlp.router" not in d and "l0.norm2" in d
    assert "loop.step" not in declare_model(spec_of(tn.U)) and "l1.mlp.shared.gate" not in declare_model(spec_of(tn.T))


@pytest.mark.parametrize("edit, word", [
    (lambda c: c["layers"][0].__setitem__("type", "conv"), "known mixer"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("heads", 0), "positive"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("rot_dim", 8), "unknown key"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("mask", {"size": 3}), "unknown key"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 9), "router.top"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("scale", 2.0), "unknown key"),
    (lambda c: c["layers"][0]["mlp"]["shared"].__setitem__("ff", 0), "shared"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "kind"),
    (lambda c: c["embedding"]["bigram"].__setitem__("buckets", 0), "buckets"),
    (lambda c: c["loop"].__setitem__("stop", 9), "loop"),
    (lambda c: c["norm"].__setitem__("eps", 0), "eps"),
    (lambda c: c.pop("width"), "width"),
])
def test_a_configuration_that_cannot_be_is_refused(edit, word):
    cfg = copy.deepcopy(tn.S)
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        spec_of(cfg)
    assert word in str(e.value)


def test_random_folders_hold_the_declared_tensors(nirozen_folders):
    for name in tn.CONFIGS:
        cfg, w = read_model(nirozen_folders[name])
        d = declare_model(spec_of(cfg))
        assert set(w) == set(d)
        assert all(tuple(w[k].shape) == tuple(d[k].shape) for k in d)
        assert abs(float(w["final.norm"].mean())) < 0.2          # stored around zero
        assert abs(float(w["l0.mix.dq.norm"].mean()) - 1.0) < 0.2    # stored around one


def test_a_norm_with_an_offset_adds_it_once():
    ctx = BuildContext(device=torch.device("cpu"), dtype=torch.float32, max_positions=1)
    stored = torch.tensor([0.25, -0.5, 0.0])
    for gain, t in (("vector", stored), ("scalar", torch.tensor(0.5))):
        n = build_norm(NormSpec(3, 1e-5, gain=gain, gain_offset=1.0), ctx)
        n.bind({"weight": t})
        assert torch.equal(n.weight, (t + 1.0).expand(3))
        assert n.declare()["weight"].init == "normal"
    old = build_norm(NormSpec(3, 1e-5), ctx)
    old.bind({"weight": stored})
    assert old.weight is stored and old.declare()["weight"].init == "gain"


# ---- the plain implementation's own identities ----
def test_the_pair_table_rows():
    ids = torch.tensor([4, 1, 1, 5])
    assert plain.pair_rows(ids, 7, 3, 5).tolist() == [7, (4 * 3 + 1 * 5) % 7, (1 * 3 + 1 * 5) % 7, (1 * 3 + 5 * 5) % 7]


def test_the_position_vector():
    for width in (2, 7, 10):
        v = plain.place_vectors(5, width, torch.float64)
        for p in range(5):
            for i in range(width // 2):
                a = p * 10000.0 ** (-2.0 * i / width)
                assert abs(float(v[p, 2 * i]) - math.sin(a)) < 1e-12 and abs(float(v[p, 2 * i + 1]) - math.cos(a)) < 1e-12
        assert v[0, 0::2].abs().max() == 0 and bool((v[0, 1::2] == 1).all())
    # the product's frequencies are the same ones, counted in turns
    turns = sinusoid_turns(7, 10000.0, "cpu")
    torch.testing.assert_close(torch.sin(2 * math.pi * turns * 4)[:3], plain.place_vectors(5, 7, torch.float64)[4, 0:6:2])
    assert turns.dtype == torch.float64 and turns.shape == (4,)
    with pytest.raises(ValueError):
        sinusoid_turns(8, 0.0, "cpu")


def test_a_sink_is_one_more_key_without_a_value():
    torch.manual_seed(1)
    q, k, v = (torch.randn(9, 2, 4, dtype=torch.float64) for _ in range(3))
    sink = torch.tensor([0.7, -1.3], dtype=torch.float64)
    got = plain.causal_sink_attention(q, k, v, 0.5, sink)
    for i in (0, 3, 8):
        for h in range(2):
            s = torch.cat([(k[:i + 1, h] @ q[i, h]) * 0.5, sink[h:h + 1]])       # the sink is not scaled
            p = torch.softmax(s, -1)
            torch.testing.assert_close(got[i, h], p[:-1] @ v[:i + 1, h])
    # a sink far below every score is no sink; one far above every score takes everything
    low = plain.causal_sink_attention(q, k, v, 0.5, torch.full((2,), -700.0, dtype=torch.float64))
    torch.testing.assert_close(low[0], v[0])
    assert float(plain.causal_sink_attention(q, k, v, 0.5, torch.full((2,), 60.0, dtype=torch.float64)).abs().max()) < 1e-20


def test_gains_are_stored_less_one():
    x = torch.randn(4, 6, dtype=torch.float64)
    torch.testing.assert_close(plain.centred_norm(x, torch.zeros(6, dtype=torch.float64), 1e-5), plain.rms(x, 1e-5))
    torch.testing.assert_close(plain.centred_norm(x, torch.full((6,), -1.0, dtype=torch.float64), 1e-5), torch.zeros_like(x))
    assert abs(float((plain.rms(x, 0.0)[0] ** 2).mean()) - 1.0) < 1e-12


def test_the_carried_form_is_the_same_attention(nirozen_folders):
    """Scores against the latents with the key up-projection moved onto the query, values up-projected behind the weighted
    sum: what the cached form relies on."""
    cfg, w = read_model(nirozen_folders["S"])
    w = {k: v.double() for k, v in w.items()}
    m, p, eps = cfg["layers"][0]["mixer"], "l0.mix.", cfg["norm"]["eps"]
    h = torch.randn(11, cfg["width"], dtype=torch.float64)
    want = plain.latent_attention(h, w, p, m, eps)
    H, T = m["heads"], 11
    q = (plain.rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"] @ w[p + "uq"].T).reshape(T, H, m["dim"])
    c = plain.rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    q_lat = torch.einsum("thd,hdr->thr", q, w[p + "uk"].reshape(H, m["dim"], -1))
    o = plain.causal_sink_attention(q_lat, c[:, None].expand(T, H, -1), c[:, None].expand(T, H, -1), m["scale"], w[p + "sink"])
    v = torch.einsum("thr,hvr->thv", o, w[p + "uv"].reshape(H, m["vdim"], -1)).reshape(T, -1)
    torch.testing.assert_close((v * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T, want)


def test_the_chosen_experts_and_their_weights():
    h = torch.tensor([[1.0, 0.0], [0.0, 2.0]], dtype=torch.float64)
    w = {"router": torch.tensor([[1.0, 0.0], [0.0, 1.0], [0.5, 0.5]], dtype=torch.float64),
         "router.b": torch.tensor([0.0, 0.0, 10.0], dtype=torch.float64)}
    idx, wt, margin = plain.expert_choice(h, w, "", {"router": {"experts": 3, "top": 2}})
    assert idx.tolist() == [[2, 0], [2, 1]]                # the bias is part of the logit: it moves the choice ...
    torch.testing.assert_close(wt, torch.softmax(torch.tensor([[10.5, 1.0], [11.0, 2.0]], dtype=torch.float64), -1))    # ... and the weights
    assert bool((margin > 0).all())


def test_whole_model_runs_and_greedy_generation_repeats(nirozen_folders):
    cfg, w = read_model(nirozen_folders["S"])
    ids = [5, 9, 200, 1, 1, 77, 180, 4]
    logits, stream = plain.forward(cfg, w, ids, torch.float64, keep_stream=True)
    assert logits.shape == (8, 211) and stream.shape == (5, 8, 75) and bool(torch.isfinite(logits).all())
    again = plain.forward(cfg, w, ids + [3, 3], torch.float64)      # causal: a longer sequence leaves the earlier rows alone
    torch.testing.assert_close(again[:8], logits)
    out = plain.greedy_generate(cfg, w, ids[:3], 4)
    assert len(out) == 4 and out == plain.greedy_generate(cfg, w, ids[:3], 4)
    # every mechanism moves the logits by far more than a tolerance of the tests
    for change in (lambda k, v: v - 50 if k.endswith(".sink") else v, lambda k, v: v * 0 if k == "bigram" else v,
                   lambda k, v: v * 0 if k == "loop.step" else v, lambda k, v: v * 0 if k.endswith("router.b") else v,
                   lambda k, v: v * 0 if ".shared.down" in k else v, lambda k, v: v * 0 if k.endswith("norm1") else v):
        other = plain.forward(cfg, {k: change(k, v) for k, v in w.items()}, ids, torch.float64)
        assert float((other - logits).abs().max()) > 0.03
