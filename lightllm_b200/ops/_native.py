"""ctypes loader for the in-tree native libraries.

``kernels()`` returns ``libllb_kernels.so`` (sm_100a CUDA kernels), ``runtime()`` returns
``libllb_runtime.so`` (host C++: shm atomics, slot allocator, radix tree).  The CUDA path never
falls back silently.  In a checkout without built libraries (and unless LLB_AUTOBUILD=0) the kernels are
compiled on first use, one library per source file, so a program compiles what it calls and no more;
`prepare` compiles a known set side by side.  `python -m lightllm_b200.build` builds everything into one library.
"""
from __future__ import annotations

import ctypes
import os
import re
from pathlib import Path

import torch

_LIB_DIR = Path(__file__).resolve().parent.parent / "_lib"
_kernels = None
_runtime = None


class NativeError(RuntimeError):
    pass


_ERR_NAMES = {-1: "bad argument", -2: "unsupported shape/dtype", -3: "size beyond the stated maximum", -4: "driver entry point unavailable"}


def check(rc: int, what: str) -> None:
    if rc == 0:
        return
    if rc < 0:
        raise NativeError(f"{what}: {_ERR_NAMES.get(rc, rc)}")
    raise NativeError(f"{what}: CUDA error {rc}")


def _load(name: str):
    path = _LIB_DIR / name
    if not path.exists():
        if os.environ.get("LLB_AUTOBUILD", "1") == "1":
            from .. import build as _b

            if name == "libllb_runtime.so":
                _b.build_runtime(verbose=False)
    if not path.exists():
        raise NativeError(f"{path} is missing: run `python -m lightllm_b200.build`")
    return ctypes.CDLL(str(path))


def debug_bounds_enabled() -> bool:
    return os.environ.get("LLB_DEBUG_BOUNDS", "0") == "1"


class UnitLibraries:
    """Stands in for libllb_kernels.so: looks an entry point up in the source that exports it and loads that unit's
    library, compiling it if need be."""

    def __init__(self):
        from .. import build

        self._build = build
        self._unit_of = {}
        self._libs = {}
        pat = re.compile(r"LLB_EXPORT\s+\w+\s*\*?\s*(llb_\w+)\s*\([^;{]*\)\s*\{")   # definitions only
        text = {src.stem: src.read_text() for src in build.CSRC.glob("*.cu")}
        for unit, body in text.items():
            for name in pat.findall(body):
                self._unit_of[name] = unit
        # units whose entry points a unit calls: linked into its library
        code = {u: re.sub(r"//[^\n]*", "", b) for u, b in text.items()}
        self._needs = {u: sorted({self._unit_of[n] for n in re.findall(r"\b(llb_\w+)\s*\(", b)
                                  if self._unit_of.get(n, u) != u}) for u, b in code.items()}

    def prepare(self, units):
        self._build.build_units(units, self._needs)

    def _load_unit(self, unit):
        if unit not in self._libs:
            self._libs[unit] = ctypes.CDLL(str(self._build.build_units([unit], self._needs)[0]))
        return self._libs[unit]

    def __getattr__(self, name):
        if not name.startswith("llb_"):
            raise AttributeError(name)
        unit = self._unit_of.get(name)
        if unit is None:
            raise AttributeError(f"no kernel source exports {name}")
        fn = getattr(self._load_unit(unit), name)
        setattr(self, name, fn)
        return fn


def prepare(units=None):
    """Compiles the named csrc units side by side when there is no built library (None: the whole library)."""
    if units is None or have_kernels() or debug_bounds_enabled() or os.environ.get("LLB_AUTOBUILD", "1") != "1":
        kernels()
    else:
        kernels().prepare(units)


def kernels():
    global _kernels
    if _kernels is None:
        if debug_bounds_enabled():   # the build with index checks (csrc/common.cuh)
            if not (_LIB_DIR / "libllb_kernels_dbg.so").exists():
                from .. import build as _b

                _b.build_kernels(verbose=False, debug_bounds=True)
            _kernels = _load("libllb_kernels_dbg.so")
        elif not have_kernels() and os.environ.get("LLB_AUTOBUILD", "1") == "1":
            _kernels = UnitLibraries()
        else:
            _kernels = _load("libllb_kernels.so")
    return _kernels


_DEBUG_UNITS = ("ops_basic", "attention", "attention_tc", "latent_attn", "mla", "moe", "norm_shift", "rms_stream")


def set_debug_bounds(pool_slots: int = 0, req_rows: int = 0, r2t_cols: int = 0, num_experts: int = 0, status=None):
    """Declares the table sizes the checked build compares indices with (0 = unchecked) and the int32 device word
    that receives the code of the first violation.  A no-op in the regular build."""
    if not debug_bounds_enabled():
        return False
    lib = kernels()
    for unit in _DEBUG_UNITS:
        fn = getattr(lib, f"llb_debug_set_bounds_{unit}")
        check(fn(ctypes.c_int(pool_slots), ctypes.c_int(req_rows), ctypes.c_int(r2t_cols), ctypes.c_int(num_experts),
                 ptr(status)), f"debug_set_bounds_{unit}")
    return True


def runtime():
    global _runtime
    if _runtime is None:
        _runtime = _load("libllb_runtime.so")
    return _runtime


def have_kernels() -> bool:
    return (_LIB_DIR / "libllb_kernels.so").exists()


# ---- argument helpers ----
c_void_p = ctypes.c_void_p
c_int = ctypes.c_int
c_int64 = ctypes.c_int64
c_float = ctypes.c_float


def ptr(t):
    """Device (or pinned host) pointer of a tensor, or NULL for None."""
    if t is None:
        return c_void_p(0)
    return c_void_p(t.data_ptr())


def stream():
    return c_void_p(torch.cuda.current_stream().cuda_stream)


def i64(v):
    return c_int64(int(v))


def f32(v):
    return c_float(float(v))
