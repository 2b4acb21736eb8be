"""bin/trace_run as a user runs it: a subprocess fed JSON steps, writing <step>.f32 files."""

from __future__ import annotations

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import tiny
from plain import qwen3_plain as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def replay(folder, dtype, steps, out, max_tokens):
    proc = subprocess.Popen([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
                             "--out", str(out), "--max-tokens", str(max_tokens)],
                            stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True)
    for msg in steps:
        proc.stdin.write(json.dumps(msg) + "\n")
        proc.stdin.flush()
        line = proc.stdout.readline().strip()
        assert line == f"done {msg['step']}", line          # the next step is sent only after this one is done
    proc.stdin.close()
    assert proc.wait(timeout=120) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["B", "C"])
def test_trace_run_schedules(name, dtype, model_folders, tmp_path):
    cfg, w = plain.read_model(model_folders[name])
    V = cfg["vocab_size"]
    rng = np.random.default_rng(7)
    reqs = {r: rng.integers(0, V, size=n).tolist() for r, n in (("a", 90), ("b", 33), ("c", 5), ("d", 64))}
    ref = {r: plain.logits(cfg, w, ids, round_weights_to_bf16=(dtype == "bfloat16")) for r, ids in reqs.items()}
    steps, expect = [], {}
    # a and b and c start together with unequal prompts, then go on one token each; c ends first, then b
    cut = {"a": 50, "b": 30, "c": 3}
    steps.append({"step": 0, "entries": [{"id": r, "tokens": reqs[r][:cut[r]], "want": [cut[r] - 1] + ([0] if r == "a" else [])}
                                         for r in "abc"], "end": []})
    expect[0] = [("a", 49), ("a", 0), ("b", 29), ("c", 2)]
    k, live = 1, ["a", "b", "c"]
    while live:
        entries, wanted, ended = [], [], []
        for r in live:
            pos = cut[r] + k - 1
            want = [0] if (pos % 2 == 0 or pos == len(reqs[r]) - 1) else []
            entries.append({"id": r, "tokens": [reqs[r][pos]], "want": want})
            wanted += [(r, pos)] * len(want)
            if pos == len(reqs[r]) - 1:
                ended.append(r)
        steps.append({"step": k, "entries": entries, "end": ended})
        if wanted:
            expect[k] = wanted
        live = [r for r in live if r not in ended]
        k += 1
        if k == 12:          # a new request takes freed room while a is still running? no: a batch takes no newcomers
            pass
    # after the batch has ended, d runs whole in the room that was given back
    steps.append({"step": k, "entries": [{"id": "d", "tokens": reqs["d"], "want": list(range(64))}], "end": ["d"]})
    expect[k] = [("d", i) for i in range(64)]
    # the most tokens live at once: a, b and c grown to their ends, each rounded up to 64
    out = tmp_path / "out"
    replay(model_folders[name], dtype, steps, out, max_tokens=128 + 64 + 64)
    # the bounds of tests/test_engine_gpu.py: bfloat16 at twice the largest difference a B200 showed there
    tol = dict(rtol=1e-4, atol=2e-5) if dtype == "float32" else dict(rtol=0.0, atol=1.7e-2)
    for step, rows in expect.items():
        got = np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), V)
        want = torch.stack([ref[r][p] for r, p in rows])
        torch.testing.assert_close(torch.from_numpy(got), want, **tol)
    assert not (out / "1.f32").exists() or 1 in expect
    produced = {int(p.name[:-4]) for p in out.iterdir()}
    assert produced == set(expect)


def test_trace_run_refuses_more_tokens_than_it_was_sized_for(model_folders, tmp_path):
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": list(range(70)), "want": []}], "end": []}]
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", model_folders["A"], "--dtype",
                           "float32", "--out", str(tmp_path / "o"), "--max-tokens", "64"],
                          input=json.dumps(steps[0]) + "\n", capture_output=True, text=True, timeout=120)
    assert proc.returncode != 0 and "64" in proc.stderr


def test_trace_run_serves_a_rabadra_folder(rabadra_folders, tmp_path):
    """The same program with a Rabadra folder, float32: unequal prompts in one batch, then one token each, the shorter
    request ending first; then another request alone in the room given back."""
    import tiny_rabadra  # noqa: F401  (the fixture's configurations)
    from plain import rabadra_plain
    cfg, w = plain.read_model(rabadra_folders["A"])
    V = cfg["vocab"]
    rng = np.random.default_rng(11)
    reqs = {r: rng.integers(0, V, size=n).tolist() for r, n in (("a", 80), ("b", 9), ("c", 66))}
    ref = {r: rabadra_plain.forward(cfg, w, ids, torch.float64).float() for r, ids in reqs.items()}
    cut = {"a": 70, "b": 4}
    steps = [{"step": 0, "entries": [{"id": r, "tokens": reqs[r][:cut[r]], "want": [cut[r] - 1]} for r in "ab"], "end": []}]
    expect = {0: [("a", 69), ("b", 3)]}
    k, live = 1, ["a", "b"]
    while live:
        entries, ended = [], []
        for r in live:
            pos = cut[r] + k - 1
            entries.append({"id": r, "tokens": [reqs[r][pos]], "want": [0]})
            if pos == len(reqs[r]) - 1:
                ended.append(r)
        steps.append({"step": k, "entries": entries, "end": ended})
        expect[k] = [(r, cut[r] + k - 1) for r in live]
        live = [r for r in live if r not in ended]
        k += 1
    steps.append({"step": k, "entries": [{"id": "c", "tokens": reqs["c"], "want": [0, 64, 65]}], "end": ["c"]})
    expect[k] = [("c", 0), ("c", 64), ("c", 65)]
    out = tmp_path / "out"
    replay(rabadra_folders["A"], "float32", steps, out, max_tokens=128 + 64)
    for step, rows in expect.items():
        got = np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), V)
        torch.testing.assert_close(torch.from_numpy(got), torch.stack([ref[r][p] for r, p in rows]), rtol=2e-4, atol=2e-4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_serves_a_movalorn_folder(movalorn_folders, tmp_path, dtype):
    """The same program with a Movalorn folder: unequal prompts in one batch, then one token each past the attention
    layers' window, the shorter request ending first; then another request alone in the slot, pages and states given
    back (its first token is a sequence's first token again)."""
    import tiny_movalorn  # noqa: F401  (the fixture's configurations)
    from plain import movalorn_plain
    cfg, w = plain.read_model(movalorn_folders["K"])
    if dtype == "bfloat16":
        w = {k: (v.to(torch.bfloat16).float() if v.is_floating_point() and v.dim() > 1 and not k.endswith((".router", "loop.step")) else v)
             for k, v in w.items()}
    V = cfg["vocab"]
    rng = np.random.default_rng(12)
    reqs = {r: rng.integers(0, V, size=n).tolist() for r, n in (("a", 80), ("b", 9), ("c", 66))}
    ref = {r: movalorn_plain.forward(cfg, w, ids, torch.float64).float() for r, ids in reqs.items()}
    cut = {"a": 30, "b": 4}
    steps = [{"step": 0, "entries": [{"id": r, "tokens": reqs[r][:cut[r]], "want": [cut[r] - 1]} for r in "ab"], "end": []}]
    expect = {0: [("a", 29), ("b", 3)]}
    k, live = 1, ["a", "b"]
    while live:
        entries, ended = [], []
        for r in live:
            pos = cut[r] + k - 1
            entries.append({"id": r, "tokens": [reqs[r][pos]], "want": [0]})
            if pos == len(reqs[r]) - 1:
                ended.append(r)
        steps.append({"step": k, "entries": entries, "end": ended})
        expect[k] = [(r, cut[r] + k - 1) for r in live]
        live = [r for r in live if r not in ended]
        k += 1
    steps.append({"step": k, "entries": [{"id": "c", "tokens": reqs["c"], "want": [0, 36, 37, 65]}], "end": ["c"]})
    expect[k] = [("c", 0), ("c", 36), ("c", 37), ("c", 65)]
    out = tmp_path / "out"
    # the bare count of live tokens (80 + 9): the two requests' part-empty last pages are the runner's business
    replay(movalorn_folders["K"], dtype, steps, out, max_tokens=89)
    tol = dict(rtol=2e-4, atol=2e-4) if dtype == "float32" else dict(rtol=0.0, atol=0.3)
    wrong = total = 0
    for step, rows in expect.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), V).copy())
        want = torch.stack([ref[r][p] for r, p in rows])
        assert bool(torch.isfinite(got).all())
        if dtype == "float32":
            torch.testing.assert_close(got, want, **tol)
        else:       # a token that chooses its experts by a hair may part ways with the plain code in bfloat16: count rows
            wrong += int(((got - want).abs().amax(-1) > tol["atol"]).sum())
            total += len(rows)
    assert wrong <= total // 10


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_serves_a_fekitar_folder(fekitar_folders, tmp_path, dtype):
    """The same program with a Fekitar folder: unequal prompts in one batch, then one token each past the windows, the
    shorter request ending first; then another request alone in the slot, pages, states and tails given back."""
    from plain import fekitar_plain
    cfg, w = plain.read_model(fekitar_folders["R"])
    if dtype == "bfloat16":
        w = {k: (v.to(torch.bfloat16).float() if v.is_floating_point() and v.dim() > 1 and not k.endswith((".router", ".mix", ".conv", ".shared.sg")) else v)
             for k, v in w.items()}
    V = cfg["vocab"]
    rng = np.random.default_rng(13)
    reqs = {r: rng.integers(0, V, size=n).tolist() for r, n in (("a", 80), ("b", 9), ("c", 66))}
    ref = {r: fekitar_plain.forward(cfg, w, torch.tensor(ids), torch.float64)[0].float() for r, ids in reqs.items()}
    cut = {"a": 30, "b": 4}
    steps = [{"step": 0, "entries": [{"id": r, "tokens": reqs[r][:cut[r]], "want": [cut[r] - 1]} for r in "ab"], "end": []}]
    expect = {0: [("a", 29), ("b", 3)]}
    k, live = 1, ["a", "b"]
    while live:
        entries, ended = [], []
        for r in live:
            pos = cut[r] + k - 1
            entries.append({"id": r, "tokens": [reqs[r][pos]], "want": [0]})
            if pos == len(reqs[r]) - 1:
                ended.append(r)
        steps.append({"step": k, "entries": entries, "end": ended})
        expect[k] = [(r, cut[r] + k - 1) for r in live]
        live = [r for r in live if r not in ended]
        k += 1
    steps.append({"step": k, "entries": [{"id": "c", "tokens": reqs["c"], "want": [0, 36, 37, 65]}], "end": ["c"]})
    expect[k] = [("c", 0), ("c", 36), ("c", 37), ("c", 65)]
    out = tmp_path / "out"
    replay(fekitar_folders["R"], dtype, steps, out, max_tokens=89)
    tol = dict(rtol=3e-4, atol=3e-4) if dtype == "float32" else dict(rtol=0.0, atol=0.6)
    wrong = total = 0
    for step, rows in expect.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), V).copy())
        want = torch.stack([ref[r][p] for r, p in rows])
        assert bool(torch.isfinite(got).all())
        if dtype == "float32":
            torch.testing.assert_close(got, want, **tol)
        else:       # a token that chooses its experts by a hair may part ways with the plain code in bfloat16: count rows
            wrong += int(((got - want).abs().amax(-1) > tol["atol"]).sum())
            total += len(rows)
    assert wrong <= total // 10


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_serves_a_nirozen_folder(nirozen_folders, tmp_path, dtype):
    """The same program with a Nirozen folder: unequal prompts in one batch, then one token each, the shorter request
    ending first; then another request alone in the slot and pages given back (its first token is a sequence's first token
    again)."""
    from plain import nirozen_plain
    cfg, w = plain.read_model(nirozen_folders["S"])
    if dtype == "bfloat16":
        w = {k: (v.to(torch.bfloat16).float() if v.is_floating_point() and v.dim() > 1 and not k.endswith((".router", "loop.step")) else v)
             for k, v in w.items()}
    V = cfg["vocab"]
    rng = np.random.default_rng(14)
    reqs = {r: rng.integers(0, V, size=n).tolist() for r, n in (("a", 80), ("b", 9), ("c", 66))}
    ref = {r: nirozen_plain.forward(cfg, w, ids, torch.float64).float() for r, ids in reqs.items()}
    cut = {"a": 30, "b": 4}
    steps = [{"step": 0, "entries": [{"id": r, "tokens": reqs[r][:cut[r]], "want": [cut[r] - 1]} for r in "ab"], "end": []}]
    expect = {0: [("a", 29), ("b", 3)]}
    k, live = 1, ["a", "b"]
    while live:
        entries, ended = [], []
        for r in live:
            pos = cut[r] + k - 1
            entries.append({"id": r, "tokens": [reqs[r][pos]], "want": [0]})
            if pos == len(reqs[r]) - 1:
                ended.append(r)
        steps.append({"step": k, "entries": entries, "end": ended})
        expect[k] = [(r, cut[r] + k - 1) for r in live]
        live = [r for r in live if r not in ended]
        k += 1
    steps.append({"step": k, "entries": [{"id": "c", "tokens": reqs["c"], "want": [0, 36, 37, 65]}], "end": ["c"]})
    expect[k] = [("c", 0), ("c", 36), ("c", 37), ("c", 65)]
    out = tmp_path / "out"
    # the bare count of live tokens (80 + 9): the two requests' part-empty last pages are the runner's business
    replay(nirozen_folders["S"], dtype, steps, out, max_tokens=89)
    tol = dict(rtol=2e-4, atol=2e-4) if dtype == "float32" else dict(rtol=0.0, atol=0.3)
    wrong = total = 0
    for step, rows in expect.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), V).copy())
        want = torch.stack([ref[r][p] for r, p in rows])
        assert bool(torch.isfinite(got).all())
        if dtype == "float32":
            torch.testing.assert_close(got, want, **tol)
        else:       # a token that chooses its experts by a hair may part ways with the plain code in bfloat16: count rows
            wrong += int(((got - want).abs().amax(-1) > tol["atol"]).sum())
            total += len(rows)
    assert wrong <= total // 10


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_serves_a_levolix_folder(levolix_folders, tmp_path, dtype):
    """The same program with a Levolix folder: unequal prompts in one batch, then one token each past the chunks, the
    shorter request ending first; then another request alone in the slot, pages, states and tails given back."""
    from plain import levolix_plain
    folder = levolix_folders["F steady" if dtype == "bfloat16" else "F"]
    cfg, w = plain.read_model(folder)
    if dtype == "bfloat16":
        w = {k: (v.to(torch.bfloat16).float() if v.is_floating_point() and v.dim() > 1 and not k.endswith((".router", ".conv")) else v)
             for k, v in w.items()}
    V = cfg["vocab"]
    rng = np.random.default_rng(13)
    reqs = {r: rng.integers(0, V, size=n).tolist() for r, n in (("a", 80), ("b", 9), ("c", 66))}
    ref = {r: levolix_plain.forward(cfg, w, torch.tensor(ids), torch.float64)[0].float() for r, ids in reqs.items()}
    cut = {"a": 30, "b": 4}
    steps = [{"step": 0, "entries": [{"id": r, "tokens": reqs[r][:cut[r]], "want": [cut[r] - 1]} for r in "ab"], "end": []}]
    expect = {0: [("a", 29), ("b", 3)]}
    k, live = 1, ["a", "b"]
    while live:
        entries, ended = [], []
        for r in live:
            pos = cut[r] + k - 1
            entries.append({"id": r, "tokens": [reqs[r][pos]], "want": [0]})
            if pos == len(reqs[r]) - 1:
                ended.append(r)
        steps.append({"step": k, "entries": entries, "end": ended})
        expect[k] = [(r, cut[r] + k - 1) for r in live]
        live = [r for r in live if r not in ended]
        k += 1
    steps.append({"step": k, "entries": [{"id": "c", "tokens": reqs["c"], "want": [0, 36, 37, 65]}], "end": ["c"]})
    expect[k] = [("c", 0), ("c", 36), ("c", 37), ("c", 65)]
    out = tmp_path / "out"
    replay(folder, dtype, steps, out, max_tokens=89)
    tol = dict(rtol=3e-4, atol=3e-3) if dtype == "float32" else dict(rtol=0.0, atol=1.2)
    for step, rows in expect.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), V).copy())
        want = torch.stack([ref[r][p] for r, p in rows])
        assert bool(torch.isfinite(got).all())
        torch.testing.assert_close(got, want, **tol)
