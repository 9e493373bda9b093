"""What the programs in bin/ share: the package with a library that holds the model's decoder, compiled if need be."""
import importlib.util
import json
import os

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PKG_DIR = os.path.join(ROOT, "amd-incstinct-labs_b200")
E_DTYPE = -2


def _load(name, path, **kw):
    spec = importlib.util.spec_from_file_location(name, path, **kw)
    mod = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(mod)
    return mod


def architecture(model_dir):
    """config.json's "architecture"; a directory without config.json is in the Llama export format."""
    path = os.path.join(model_dir, "config.json")
    if not os.path.exists(path):
        return "Llama"
    with open(path) as f:
        return json.load(f)["architecture"]


def package_for(model_dir):
    build = _load("b200p_build", os.path.join(PKG_DIR, "build.py"))
    arch = architecture(model_dir)
    if arch not in build.DECODERS:
        raise ValueError(f"unknown architecture {arch!r}; known: {', '.join(sorted(build.DECODERS))}")
    path = build.build_decoder(arch)
    pkg = _load("amd_incstinct_labs_b200", os.path.join(PKG_DIR, "__init__.py"), submodule_search_locations=[PKG_DIR])
    pkg.load_library(path, whole=path == build.LIB)
    return pkg
