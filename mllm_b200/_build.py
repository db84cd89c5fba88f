"""Build / load the native extensions in-tree.

The extensions live under ``mllm_b200/csrc``:

* ``mllm_b200_C``    — the sm_100a CUDA kernels of every decoder plus their PyTorch binding;
* ``mllm_b200_R``    — gated delta rule;
* ``mllm_b200_A``    — latent attention;
* ``mllm_b200_L``    — lightning attention (linear attention with a fixed decay per head);
* ``mllm_b200_E``    — mixtures of experts;
* ``mllm_b200_X``    — 4-bit weights, vision towers, tensor- and expert-parallel exchange;
* ``mllm_b200_host`` — host-only C++ (radix tree, page allocator, ``.mllm`` file reader).

A CUDA module other than the first is loaded, and where it is missing compiled, when one of its functions is first
called: a model compiles what it needs.

They are compiled with ``torch.utils.cpp_extension.load`` into ``mllm_b200/_ext`` so the
shared objects sit beside the package (not in a user cache) and travel with the source
tree.  A content hash of the sources is stored next to each ``.so``; at import time a
``.so`` whose hash matches is loaded directly, without invoking ninja.
"""

from __future__ import annotations

import hashlib
import importlib.util
import os
import re
import sys
import threading
from pathlib import Path
from types import ModuleType
from typing import Dict, List, Optional

_PKG = Path(__file__).resolve().parent
_CSRC = _PKG / "csrc"
_OUT = _PKG / "_ext"

CUDA_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17", "--expt-relaxed-constexpr",
    "-Xptxas", "-v",
]
CXX_FLAGS = ["-O3", "-std=c++17"]
# the libstdc++ that torch uses, also where the compiler would link its own copy statically: with two copies in a process
# the first number that is formatted into an error message crashes instead of raising
LD_FLAGS = ["-l:libstdc++.so.6"]

_COMMON = ["bindings_common.h", "common.cuh", "kernels.h", "mma.cuh", "row.cuh"]

EXTENSIONS: Dict[str, Dict[str, List[str]]] = {
    "mllm_b200_C": {
        "sources": ["bindings.cpp", "runtime.cu", "elementwise.cu", "row_ops.cu", "depth.cu", "gemm_tcgen05.cu", "gemm_smallm.cu", "attention.cu",
                    "attention_rows.cu", "sampling.cu", "no_alloc.cu"],
        "headers": _COMMON + ["no_alloc.h"],
        "cuda": True,
    },
    "mllm_b200_R": {
        "sources": ["bindings_recurrent.cpp", "runtime.cu", "gdn.cu", "gdn_chunk.cu", "gdn_channel.cu"],
        "headers": _COMMON,
        "cuda": True,
    },
    "mllm_b200_A": {
        "sources": ["bindings_latent.cpp", "runtime.cu", "latent.cu"],
        "headers": _COMMON,
        "cuda": True,
    },
    "mllm_b200_L": {
        "sources": ["bindings_lightning.cpp", "runtime.cu", "lightning.cu"],
        "headers": _COMMON,
        "cuda": True,
    },
    "mllm_b200_E": {
        "sources": ["bindings_moe.cpp", "runtime.cu", "moe.cu"],
        "headers": _COMMON,
        "cuda": True,
    },
    "mllm_b200_X": {
        "sources": ["bindings_extra.cpp", "runtime.cu", "comm.cu", "ep_a2a.cu", "gemm_w4a16.cu", "gemm_smallm_w4.cu", "vision.cu"],
        "headers": _COMMON,
        "cuda": True,
    },
    "mllm_b200_host": {
        "sources": ["host/host_bindings.cpp", "host/radix_tree.cpp", "host/page_allocator.cpp", "host/mllm_file.cpp", "host/cpu_oracle.cpp", "host/symm_heap.cpp"],
        "headers": ["host/radix_tree.h", "host/page_allocator.h", "host/mllm_file.h", "host/cpu_oracle.h", "host/symm_heap.h"],
        "cuda": False,
    },
}

_loaded: Dict[str, ModuleType] = {}
_lock = threading.Lock()


def cuda_modules() -> List[str]:
    """The CUDA extension modules, the one of every decoder first."""
    return [n for n, spec in EXTENSIONS.items() if spec["cuda"]]


def module_functions(name: str) -> List[str]:
    """Names of the functions a CUDA module binds, read from its binding source (the first of its sources)."""
    return re.findall(r'm\.def\("(\w+)"', (_CSRC / EXTENSIONS[name]["sources"][0]).read_text())


def _existing(names: List[str]) -> List[Path]:
    return [(_CSRC / n) for n in names if (_CSRC / n).exists()]


def _source_hash(name: str) -> str:
    spec = EXTENSIONS[name]
    h = hashlib.sha256()
    for p in sorted(_existing(spec["sources"]) + _existing(spec["headers"])):
        h.update(p.name.encode())
        h.update(p.read_bytes())
    h.update(" ".join((CUDA_FLAGS if spec["cuda"] else CXX_FLAGS) + LD_FLAGS).encode())
    return h.hexdigest()


def _so_path(name: str) -> Path:
    return _OUT / name / f"{name}.so"


def _hash_path(name: str) -> Path:
    return _OUT / name / "source.sha256"


def _import_so(name: str) -> ModuleType:
    import torch  # noqa: F401  (the extension links against libtorch)

    spec = importlib.util.spec_from_file_location(name, _so_path(name))
    mod = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(mod)
    sys.modules[name] = mod
    return mod


def is_built(name: str) -> bool:
    return _so_path(name).exists() and _hash_path(name).exists() and _hash_path(name).read_text().strip() == _source_hash(name)


def build_extension(name: str, verbose: bool = False) -> ModuleType:
    """Compile ``name`` (if its sources changed) and import it."""
    from torch.utils import cpp_extension

    spec = EXTENSIONS[name]
    out = _OUT / name
    out.mkdir(parents=True, exist_ok=True)
    sources = [str(p) for p in _existing(spec["sources"])]
    os.environ.setdefault("MAX_JOBS", str(min(8, os.cpu_count() or 1)))
    mod = cpp_extension.load(
        name=name,
        sources=sources,
        extra_cflags=CXX_FLAGS,
        extra_cuda_cflags=CUDA_FLAGS if spec["cuda"] else None,
        extra_include_paths=[str(_CSRC)],
        extra_ldflags=list(LD_FLAGS),      # load() appends to it
        build_directory=str(out),
        with_cuda=spec["cuda"],
        verbose=verbose,
    )
    _hash_path(name).write_text(_source_hash(name))
    sys.modules[name] = mod
    return mod


def load_extension(name: str, build_if_missing: bool = True) -> Optional[ModuleType]:
    """Import ``name`` from the in-tree ``.so``; compile first when it is missing or stale."""
    with _lock:
        if name in _loaded:
            return _loaded[name]
        mod: Optional[ModuleType] = None
        if is_built(name):
            mod = _import_so(name)
        elif build_if_missing:
            mod = build_extension(name)
        if mod is not None:
            _loaded[name] = mod
        return mod


def build_all(verbose: bool = False) -> None:
    for name in EXTENSIONS:
        if not _existing(EXTENSIONS[name]["sources"]):
            continue
        if not is_built(name):
            build_extension(name, verbose=verbose)
        load_extension(name)


if __name__ == "__main__":
    build_all(verbose="-v" in sys.argv)
    print("built:", {n: str(_so_path(n)) for n in EXTENSIONS})
