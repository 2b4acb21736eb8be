"""Shared test set-up: the ``gpu`` marker, import paths, the tiny configurations and model folders."""

from __future__ import annotations

import os
import sys

import pytest

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
for p in (ROOT, os.path.dirname(os.path.abspath(__file__))):
    if p not in sys.path:
        sys.path.insert(0, p)


def pytest_configure(config):
    config.addinivalue_line("markers", "gpu: needs an NVIDIA GPU (run with -m gpu on a B200)")


def pytest_collection_modifyitems(config, items):
    import torch
    if torch.cuda.is_available():
        return
    skip = pytest.mark.skip(reason="no CUDA device here")
    for item in items:
        if "gpu" in item.keywords:
            item.add_marker(skip)


@pytest.fixture(scope="session")
def model_folders(tmp_path_factory):
    """Model folders of the tiny configurations, float32 weights, made once per session."""
    import torch

    import tiny
    from sleuth_b200.weights.random_init import write_random_model
    out = {}
    for name, cfg in tiny.CONFIGS.items():
        d = tmp_path_factory.mktemp(f"model_{name}")
        write_random_model(d, cfg, seed=tiny.SEEDS[name], dtype=torch.float32)
        out[name] = str(d)
    return out


@pytest.fixture(scope="session")
def lezepel_folders(tmp_path_factory):
    """Model folders of the tiny Lezepel configurations, float32 weights, made once per session."""
    import torch

    import tiny_lezepel
    from sleuth_b200.weights.random_init import write_random_model
    out = {}
    for name, cfg in tiny_lezepel.CONFIGS.items():
        d = tmp_path_factory.mktemp(f"lezepel_{name}")
        write_random_model(d, cfg, seed=tiny_lezepel.SEEDS[name], dtype=torch.float32, std=tiny_lezepel.STD)
        tiny_lezepel.spread_router_biases(d)
        out[name] = str(d)
    return out


@pytest.fixture(scope="session")
def rabadra_folders(tmp_path_factory):
    """Model folders of the tiny Rabadra configurations, float32 weights, made once per session."""
    import torch

    import tiny_rabadra
    from sleuth_b200.weights.random_init import write_random_model
    out = {}
    for name, cfg in tiny_rabadra.CONFIGS.items():
        d = tmp_path_factory.mktemp(f"rabadra_{name}")
        write_random_model(d, cfg, seed=tiny_rabadra.SEEDS[name], dtype=torch.float32, std=tiny_rabadra.STD)
        tiny_rabadra.sharpen(d, round_router=name in ("C", "D"))
        out[name] = str(d)
    return out


@pytest.fixture(scope="session")
def fekitar_folders(tmp_path_factory):
    """Model folders of the tiny Fekitar configurations, float32 weights, made once per session."""
    import torch

    import tiny_fekitar
    from sleuth_b200.weights.random_init import write_random_model
    out = {}
    for name, cfg in tiny_fekitar.CONFIGS.items():
        d = tmp_path_factory.mktemp(f"fekitar_{name}")
        write_random_model(d, cfg, seed=tiny_fekitar.SEEDS[name], dtype=torch.float32, std=tiny_fekitar.STD)
        tiny_fekitar.sharpen(d)
        out[name] = str(d)
    return out


@pytest.fixture(scope="session")
def movalorn_folders(tmp_path_factory):
    """Model folders of the tiny Movalorn configurations, float32 weights, made once per session."""
    import torch

    import tiny_movalorn
    from sleuth_b200.weights.random_init import write_random_model
    out = {}
    for name, cfg in tiny_movalorn.CONFIGS.items():
        d = tmp_path_factory.mktemp(f"movalorn_{name}")
        write_random_model(d, cfg, seed=tiny_movalorn.SEEDS[name], dtype=torch.float32, std=tiny_movalorn.STD)
        tiny_movalorn.sharpen(d)
        out[name] = str(d)
    return out


@pytest.fixture(scope="session")
def nirozen_folders(tmp_path_factory):
    """Model folders of the tiny Nirozen configurations, float32 weights, made once per session."""
    import torch

    import tiny_nirozen
    from sleuth_b200.weights.random_init import write_random_model
    out = {}
    for name, cfg in tiny_nirozen.CONFIGS.items():
        d = tmp_path_factory.mktemp(f"nirozen_{name}")
        write_random_model(d, cfg, seed=tiny_nirozen.SEEDS[name], dtype=torch.float32, std=tiny_nirozen.STD)
        tiny_nirozen.sharpen(d)
        out[name] = str(d)
    return out


@pytest.fixture(scope="session")
def levolix_folders(tmp_path_factory):
    """Model folders of the tiny Levolix configurations, float32 weights, made once per session: ``name`` with choices of
    experts that depend on the token, ``name + " steady"`` with choices that the corrections alone make."""
    import torch

    import tiny_levolix
    from sleuth_b200.weights.random_init import write_random_model
    out = {}
    for name, cfg in tiny_levolix.CONFIGS.items():
        for steady in (False, True):
            d = tmp_path_factory.mktemp(f"levolix_{name}")
            write_random_model(d, cfg, seed=tiny_levolix.SEEDS[name], dtype=torch.float32, std=tiny_levolix.STD)
            tiny_levolix.sharpen(d, steady)
            out[name + " steady" * steady] = str(d)
    return out


def pytest_terminal_summary(terminalreporter):
    """The largest differences from the plain implementation that the GPU tests saw (tests/closeness.py)."""
    import closeness
    closeness.report(terminalreporter.write_line)
