"""Compiling the kernel library for sm_100a and loading it.

The sources under this folder are compiled with nvcc, either all of them into one shared library,
``_build/libcitlali_b200.so`` beside them (``build()``; what a C or C++ program links), or one by one:
:class:`Kernels` finds the source that defines an entry point the first time the entry point is asked
for, compiles that source into a shared library of its own under ``_build/single/`` and loads it, so
that a process compiles what its model needs and no more.  ``Kernels.prepare`` compiles several
sources at once, ahead of their first use.  Where the whole library is there and up to date, it is
loaded and nothing is compiled.  If ``_build`` cannot be written, a folder under the system's
temporary folder stands in.  Objects are rebuilt when their source, a header or a flag changed.
Nothing here needs a GPU: nvcc cross-compiles.
"""
from __future__ import annotations

import concurrent.futures
import ctypes
import hashlib
import os
import re
import shutil
import subprocess
import sys
import tempfile
import threading
import time

from ..errors import CitlaliError

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_NAME = "libcitlali_b200.so"
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr"]
_lock = threading.Lock()
_lib = None


def _say(message):
    print(f"[citlali_b200 build] {message}", file=sys.stderr, flush=True)


def sources():
    return sorted(f for f in os.listdir(_HERE) if f.endswith(".cu"))


def _headers():
    return sorted(f for f in os.listdir(_HERE) if f.endswith((".cuh", ".h")))


def _nvcc():
    path = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.isfile(path):
        raise CitlaliError("nvcc was not found (PATH and /usr/local/cuda/bin): the kernel library cannot be "
                           "compiled, and there is no other way to run a model")
    return path


def _hash_of(files):
    h = hashlib.sha256()
    h.update(" ".join(NVCC_FLAGS).encode())
    for f in files:
        h.update(f.encode())
        with open(os.path.join(_HERE, f), "rb") as fh:
            h.update(fh.read())
    return h.hexdigest()


def _digest():
    return _hash_of(sources() + _headers())


def _build_dir():
    preferred = os.path.join(_HERE, "_build")
    try:
        os.makedirs(preferred, exist_ok=True)
        probe = os.path.join(preferred, f".write_probe_{os.getpid()}")
        with open(probe, "w"):
            pass
        os.remove(probe)
        return preferred
    except OSError:
        fallback = os.path.join(tempfile.gettempdir(), f"citlali_b200_build_{os.getuid()}")
        os.makedirs(fallback, exist_ok=True)
        return fallback


def library_path():
    return os.path.join(_build_dir(), LIB_NAME)


def _stamped(path, digest) -> bool:
    """Whether ``path`` was made from what ``digest`` stands for."""
    try:
        with open(path + ".sha256") as f:
            return os.path.isfile(path) and f.read().strip() == digest
    except OSError:
        return False


def _stamp(path, digest):
    tmp = f"{path}.sha256.{os.getpid()}.tmp"
    with open(tmp, "w") as f:
        f.write(digest)
    os.replace(tmp, path + ".sha256")


def _compile(stems, force=False, verbose=True):
    """The objects of ``stems`` (a source's name without .cu), compiled side by side where they are stale: {stem: (path, digest)}."""
    nvcc, out_dir = _nvcc(), _build_dir()
    headers = _headers()
    out = {}
    stale = []
    for stem in stems:
        obj, digest = os.path.join(out_dir, stem + ".o"), _hash_of([stem + ".cu"] + headers)
        out[stem] = (obj, digest)
        if force or not _stamped(obj, digest):
            stale.append(stem)
    if not stale:
        return out
    if verbose:
        _say(f"compiling {len(stale)} CUDA source{'s' if len(stale) > 1 else ''} for sm_100a into {out_dir} (first use, or the sources changed)")
    t0 = time.time()

    def compile_one(stem):
        obj, digest = out[stem]
        tmp = f"{obj}.{os.getpid()}.tmp.o"
        cmd = [nvcc] + NVCC_FLAGS + ["-I", _HERE, "-c", os.path.join(_HERE, stem + ".cu"), "-o", tmp]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise CitlaliError(f"nvcc failed on {stem}.cu:\n{r.stdout}\n{r.stderr}")
        os.replace(tmp, obj)
        _stamp(obj, digest)
        return stem

    done_count = 0
    with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 2)) as pool:
        pending = {pool.submit(compile_one, s) for s in stale}
        while pending:
            done, pending = concurrent.futures.wait(pending, timeout=10.0)
            for f in done:
                stem = f.result()
                done_count += 1
                if verbose:
                    _say(f"  compiled {stem}.cu ({done_count}/{len(stale)}, {time.time() - t0:.0f} s)")
            if pending and not done and verbose:
                _say(f"  still compiling ({done_count}/{len(stale)} done, {time.time() - t0:.0f} s)")
    return out


def _link(objects, path, digest):
    tmp = f"{path}.{os.getpid()}.tmp"
    r = subprocess.run([_nvcc(), "-shared", "-o", tmp] + sorted(objects), capture_output=True, text=True)
    if r.returncode != 0:
        raise CitlaliError(f"linking {os.path.basename(path)} failed:\n{r.stdout}\n{r.stderr}")
    os.replace(tmp, path)
    _stamp(path, digest)


def build(force: bool = False, verbose: bool = True) -> str:
    """Compile what is stale of the whole library; return its path."""
    lib_path, digest = library_path(), _digest()
    if not force and _stamped(lib_path, digest):
        return lib_path
    t0 = time.time()
    objects = _compile([f[:-3] for f in sources()], force, verbose)
    _link([obj for obj, _ in objects.values()], lib_path, digest)
    if verbose:
        _say(f"built {lib_path} in {time.time() - t0:.0f} s")
    return lib_path


_BASE = "elementwise"                       # holds what every other source calls (error text, launch mode)
_ALSO = {"gemm_tcgen05": ("gemm_tcgen05_pair",), "attention_decode_no_alloc": ("attention_decode",)}    # who calls whom besides
_ENTRY = re.compile(r'extern "C"[^;{]*?\b(citlali_\w+)\s*\(')


class Kernels:
    """The library's entry points as attributes.  An entry point's source is compiled and loaded when the entry point is first
    asked for; the whole library, if it is there and up to date, serves them all.  There is no other implementation of the
    kernels: a failure here is an error, never a fallback."""

    def __init__(self):
        self._whole = None
        self._loaded = {}
        self._source_of = {}
        self._lock = threading.RLock()
        if _stamped(library_path(), _digest()):
            self._whole = self._open(library_path())
            return
        for f in sources():
            with open(os.path.join(_HERE, f), encoding="utf-8") as fh:
                for symbol in _ENTRY.findall(fh.read()):
                    self._source_of[symbol] = f[:-3]

    @staticmethod
    def _open(path):
        try:
            return ctypes.CDLL(path, mode=ctypes.RTLD_GLOBAL)
        except OSError as e:
            raise CitlaliError(f"the kernel library {path} could not be loaded: {e}") from None

    def _with_callees(self, stems):
        out = []
        for stem in stems:
            for s in (_BASE,) + _ALSO.get(stem, ()) + (stem,):
                if s not in out:
                    out.append(s)
        return out

    def prepare(self, stems) -> None:
        """Compile (side by side) and load these sources and what they call, unless the whole library is loaded."""
        if self._whole is not None:
            return
        with self._lock:
            wanted = [s for s in self._with_callees(stems) if s not in self._loaded]
            if not wanted:
                return
            objects = _compile(wanted)
            folder = os.path.join(_build_dir(), "single")
            os.makedirs(folder, exist_ok=True)
            for stem in wanted:                                # callees come first
                obj, digest = objects[stem]
                path = os.path.join(folder, f"lib{stem}.so")
                if not _stamped(path, digest):
                    _link([obj], path, digest)
                self._loaded[stem] = self._open(path)

    def __getattr__(self, name):
        if name.startswith("_"):
            raise AttributeError(name)
        if self._whole is not None:
            fn = getattr(self._whole, name)
        else:
            stem = self._source_of.get(name)
            if stem is None:
                raise AttributeError(f"no kernel source defines {name}")
            self.prepare([stem])
            fn = getattr(self._loaded[stem], name)
        self.__dict__[name] = fn
        return fn


def load() -> Kernels:
    global _lib
    with _lock:
        if _lib is None:
            _lib = Kernels()
        return _lib
