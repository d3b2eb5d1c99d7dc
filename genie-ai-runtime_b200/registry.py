"""Model registry: config.json names an architecture, the registry opens it.

A model folder holds config.json ("architecture" and the architecture's own keys) and model.safetensors.  An architecture
registers one function (config, tensors, dtype) -> open_session, which loads the weights once and returns a function
(max_context, flags) -> decoder.Session.
"""
from __future__ import annotations

import json
import os


class ConfigError(ValueError):
    """A configuration, or a tensor it describes, that the named architecture cannot run."""


class DtypeError(ConfigError):
    """The architecture does not run in the requested number format."""


ARCHITECTURES = {}


def register(name, dtypes):
    """Decorator: registers an architecture and the number formats it runs in (the first is the default)."""
    def add(fn):
        ARCHITECTURES[name] = (fn, tuple(dtypes))
        return fn
    return add


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def check_config(config, dtype=None):
    """(loader, dtype) of a configuration; raises ConfigError / DtypeError without touching the weights."""
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ConfigError(f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    fn, dtypes = ARCHITECTURES[name]
    if dtype is not None and dtype not in dtypes:
        raise DtypeError(f"{name} runs in {', '.join(dtypes)}, not in {dtype}")
    return fn, dtype or dtypes[0]


def open_model(folder, dtype=None):
    """Loads a model folder; returns (config, open_session)."""
    from .safetensors import SafetensorsFile
    config = read_config(folder)
    fn, dtype = check_config(config, dtype)
    return config, fn(config, SafetensorsFile(os.path.join(folder, "model.safetensors")), dtype)
