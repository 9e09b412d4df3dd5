"""In-tree build and loading of the sm_100a CUDA extension.

The shared object lives under ``llaminar_b200/ops/_build`` (next to the sources, so a source
snapshot carries it along) together with a hash of the sources it was built from.  ``load()``
imports the existing binary when the hash still matches and rebuilds otherwise.
"""
from __future__ import annotations

import hashlib
import importlib.util
import os
import sys
from pathlib import Path

NAME = "llaminar_b200_ops"
CSRC = Path(__file__).resolve().parent / "csrc"
BUILD_DIR = Path(__file__).resolve().parent / "_build"
# kernels of models with unquantised matrices, built and loaded on their own: shared ones, latent attention, grouped-query attention,
# mixers with a recurrent state, and experts
DENSE, LATENT, GROUPED, MIXERS, EXPERTS = (f"llaminar_b200_{n}" for n in ("dense", "latent", "grouped", "mixers", "experts"))
SOURCES = {
    NAME: ["binding.cpp", "gemv.cu", "gemv_stream.cu", "gemm_tc.cu", "gemm_tc_small.cu", "attention.cu", "attention_tc.cu", "ops.cu", "gdn.cu", "moe_ep.cu", "no_alloc.cu"],
    DENSE: ["dense_binding.cpp", "dense_ops.cu"],
    LATENT: ["latent_binding.cpp", "latent_attention.cu", "latent_tc.cu"],
    GROUPED: ["grouped_binding.cpp", "grouped.cu", "attention.cu", "attention_tc.cu"],
    MIXERS: ["mixers_binding.cpp", "mixers.cu", "linear_tc.cu"],
    EXPERTS: ["experts_binding.cpp", "experts.cu", "experts_tc.cu"],
}
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "--expt-relaxed-constexpr", "-Xptxas", "-v"]

_modules: dict = {}


def _bounds_check() -> bool:
    from ..utils.env import debug_env
    return bool(debug_env().bounds_check)


def _flags() -> list[str]:
    return NVCC_FLAGS + (["-DLLM_BOUNDS_CHECK"] if _bounds_check() else [])


def _build_dir() -> Path:
    """The bounds-check variant is a build of its own (other flags, other directory), selected by LLAMINAR_BOUNDS_CHECK."""
    return BUILD_DIR.with_name("_build_bc") if _bounds_check() else BUILD_DIR


def source_hash(name: str = NAME) -> str:
    """Hash of an extension's own sources, of every header and of the compiler flags."""
    h = hashlib.sha256()
    for p in sorted(CSRC.iterdir()):
        if p.name in SOURCES[name] or p.suffix in (".cuh", ".h", ".inc"):
            h.update(p.name.encode())
            h.update(p.read_bytes())
    h.update(" ".join(_flags()).encode())
    return h.hexdigest()


def _so_path(name: str = NAME) -> Path:
    return _build_dir() / f"{name}.so"


def is_built(name: str = NAME) -> bool:
    hp = _build_dir() / f"{name}.hash"
    return _so_path(name).exists() and hp.exists() and hp.read_text().strip() == source_hash(name)


def _import_so(name: str):
    import torch  # noqa: F401  (the extension links against libtorch)
    spec = importlib.util.spec_from_file_location(name, str(_so_path(name)))
    mod = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(mod)
    sys.modules[name] = mod
    return mod


def build_extension(name: str, verbose: bool = False, force: bool = False):
    """Compile one extension for sm_100a (cross-compiles without a GPU) unless its binary is current; returns the module."""
    if not force and is_built(name):
        _modules[name] = _import_so(name)
        return _modules[name]
    from torch.utils import cpp_extension
    _build_dir().mkdir(exist_ok=True)
    os.environ.setdefault("TORCH_CUDA_ARCH_LIST", "10.0a")
    os.environ.setdefault("MAX_JOBS", str(max(1, (os.cpu_count() or 2))))
    # ninja's build file carries one extension: each has its own directory, the finished binary lands beside the others
    work = _build_dir() if name == NAME else _build_dir() / name
    work.mkdir(exist_ok=True)
    cpp_extension.load(
        name=name,
        sources=[str(CSRC / s) for s in SOURCES[name]],
        extra_cflags=["-O2", "-std=c++17"] + (["-DLLM_BOUNDS_CHECK"] if _bounds_check() else []),
        extra_cuda_cflags=_flags(),
        extra_include_paths=[str(CSRC)],
        build_directory=str(work),
        with_cuda=True,
        verbose=verbose,
        is_python_module=name == NAME,
        is_standalone=False,
    )
    if work != _build_dir():
        os.replace(work / f"{name}.so", _so_path(name))
    (_build_dir() / f"{name}.hash").write_text(source_hash(name))
    _modules[name] = sys.modules.get(name) or _import_so(name)
    return _modules[name]


def build(verbose: bool = False, force: bool = False):
    """Compile every extension; returns the main module."""
    for name in SOURCES:
        build_extension(name, verbose, force)
    return _modules[NAME]


def build_bounds_check_variant() -> None:
    """Compile the debug variant with explicit index checks (LLAMINAR_BOUNDS_CHECK=1 loads it) in a child process: the
    variant is chosen by the environment before the extension is first imported."""
    import subprocess
    env = dict(os.environ, LLAMINAR_BOUNDS_CHECK="1")
    code = "from llaminar_b200.ops import build as b; b.build()"
    subprocess.run([sys.executable, "-c", code], check=True, env=env, cwd=str(Path(__file__).resolve().parents[2]))


def load(name: str = NAME):
    """An extension module; built on first use if the in-tree binary is missing or stale."""
    if name not in _modules:
        build_extension(name)
    return _modules[name]


def so_path(name: str = NAME) -> str:
    return str(_so_path(name))


if __name__ == "__main__":
    build(verbose=True, force="--force" in sys.argv)
    print("built", _so_path())
