import os
import sys

import pytest

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
for p in (ROOT, os.path.dirname(os.path.abspath(__file__))):
    if p not in sys.path:
        sys.path.insert(0, p)


def pytest_configure(config):
    config.addinivalue_line("markers", "gpu: needs a CUDA device (run with -m gpu on a B200)")


def pytest_collection_modifyitems(config, items):
    import torch
    if torch.cuda.is_available():
        return
    skip = pytest.mark.skip(reason="no CUDA device")
    for item in items:
        if "gpu" in item.keywords:
            item.add_marker(skip)


@pytest.fixture(scope="session")
def folders(tmp_path_factory):
    """Factory: (config name, dtype) -> model folder with random weights, made once per session."""
    from helpers import (CONFIGS, DUBODRA_CONFIGS, FIGALIX_CONFIGS, GEDILORN_CONFIGS, LUDUSUN_CONFIGS, RIFIZEN_CONFIGS, VILULORN_CONFIGS,
                         write_dubodra, write_figalix, write_gedilorn, write_ludusun, write_rifizen, write_tiny, write_vilulorn)
    made = {}

    def get(name: str, dtype: str = "float32") -> str:
        key = (name, dtype)
        if key not in made:
            d = tmp_path_factory.mktemp(f"model_{name}_{dtype}")
            if name in DUBODRA_CONFIGS:
                write_dubodra(DUBODRA_CONFIGS[name], str(d), dtype)
            elif name in GEDILORN_CONFIGS:
                write_gedilorn(GEDILORN_CONFIGS[name], str(d), dtype)
            elif name in LUDUSUN_CONFIGS:
                write_ludusun(LUDUSUN_CONFIGS[name], str(d), dtype)
            elif name in FIGALIX_CONFIGS:
                write_figalix(FIGALIX_CONFIGS[name], str(d), dtype)
            elif name in VILULORN_CONFIGS:
                write_vilulorn(VILULORN_CONFIGS[name], str(d), dtype)
            elif name in RIFIZEN_CONFIGS:
                write_rifizen(RIFIZEN_CONFIGS[name], str(d), dtype)
            else:
                write_tiny(CONFIGS[name], str(d), dtype)
            made[key] = str(d)
        return made[key]
    return get
