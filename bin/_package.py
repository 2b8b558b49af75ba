"""Builds the library if it is not there yet and loads the `llama.rust_b200` package (its directory name has a dot)."""
import importlib
import importlib.util
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PKG = os.path.join(ROOT, "llama.rust_b200")


def _by_path(name, path):
    spec = importlib.util.spec_from_file_location(name, path)
    mod = importlib.util.module_from_spec(spec)
    sys.modules[name] = mod
    spec.loader.exec_module(mod)
    return mod


def load(*modules):
    _by_path("b200_build", os.path.join(PKG, "build.py")).ensure()
    pkg = _by_path("llama_rust_b200", os.path.join(PKG, "__init__.py"))
    return [pkg] + [importlib.import_module("llama_rust_b200." + m) for m in modules]
