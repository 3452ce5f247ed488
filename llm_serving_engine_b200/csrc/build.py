"""Compile the engine's CUDA sources for sm_100a, each into a shared library of its own.

The libraries are built with nvcc alone (no framework headers), in-tree under
``llm_serving_engine_b200/_build/``, the first time a source's kernels are
needed, and again when the source, a header that it includes or a flag changes
(the key is a hash of all three).  A model asks for the sources of its parts at
once, and they compile side by side; sources of other models are left alone.
While nvcc runs, a line is printed every few seconds so that a first call does
not look hung.  Nothing outside the package directory is written unless that
directory is read-only, in which case a per-user temporary directory is used.
"""
from __future__ import annotations

import hashlib
import os
import re
import shutil
import subprocess
import sys
import tempfile
import threading
import time
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

CSRC = Path(__file__).resolve().parent
PACKAGE = CSRC.parent
LIB_NAME = "libllmserve_b200_{source}{variant}.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
]


class BuildError(RuntimeError):
    pass


def sources() -> list[Path]:
    return sorted(CSRC.glob("*.cu"))


def _nvcc() -> str:
    for candidate in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if candidate and Path(candidate).exists():
            return candidate
    raise BuildError("nvcc not found: the CUDA kernels cannot be built (set NVCC or add it to PATH)")


_INCLUDE = re.compile(r'^\s*#include\s+"([^"]+)"', re.MULTILINE)
_EXPORT = re.compile(r'^extern "C" int\s+(lse_\w+)\s*\(|^LSE_(?:CHECK|TL)_DEFINE\((lse_\w+)\)', re.MULTILINE)


def exported_names(source: Path) -> list[str]:
    """C entry points that a source defines (the readers of the checked and tuning variants among them)."""
    return [match[1] or match[2] for match in _EXPORT.finditer(source.read_text())]


def _key(source: Path, flags: list[str]) -> str:
    """Hash of the flags, the source and every header of this directory that it includes, directly or not."""
    digest = hashlib.sha256(" ".join(flags).encode())
    waiting, seen = [source], set()
    while waiting:
        path = waiting.pop()
        if path in seen:
            continue
        seen.add(path)
        text = path.read_text()
        waiting += [CSRC / name for name in _INCLUDE.findall(text) if (CSRC / name).exists()]
    for path in sorted(seen):
        digest.update(path.name.encode())
        digest.update(path.read_bytes())
    return digest.hexdigest()[:16]


def _build_dir() -> Path:
    preferred = PACKAGE / "_build"
    try:
        preferred.mkdir(exist_ok=True)
        probe = preferred / f".write_probe_{os.getpid()}"
        probe.write_text("")
        probe.unlink()
        return preferred
    except OSError:
        fallback = Path(tempfile.gettempdir()) / f"llmserve_b200_build_{os.getuid()}"
        fallback.mkdir(parents=True, exist_ok=True)
        return fallback


def _log(message: str, verbose: bool) -> None:
    if verbose:
        print(f"[llm_serving_engine_b200] {message}", file=sys.stderr, flush=True)


def library_paths(names=None, verbose: bool = True, force: bool = False, trace: bool = False,
                  check: bool = False) -> dict[str, Path]:
    """Path of the built library of each named source (file names without the suffix; default: every source);
    compiles those that are missing or stale first, side by side.

    ``trace``: the tuning variant (``-DLSE_TRACE``), in which block 0 of every kernel records when it
    started, when its wait for the kernels before returned and when it ended; libraries of its own.
    ``check``: the checked variant (``-DLSE_CHECK``), in which every kernel compares the indices it takes
    from the step's metadata with their ranges, replaces a bad one by a safe one and records it;
    libraries of its own as well."""
    build_dir = _build_dir()
    variant = "_trace" if trace else "_check" if check else ""
    flags = NVCC_FLAGS + (["-DLSE_TRACE"] if trace else ["-DLSE_CHECK"] if check else [])
    known = {path.stem: path for path in sources()}
    found: dict[str, Path] = {}
    stale: list[tuple[str, str]] = []
    for name in sorted(known if names is None else set(names)):
        if name not in known:
            raise BuildError(f"no CUDA source {name!r}; there are {sorted(known)}")
        found[name] = build_dir / LIB_NAME.format(source=name, variant=variant)
        stamp = build_dir / f"{name}{variant}.key"
        key = _key(known[name], flags)
        if force or not found[name].exists() or not stamp.exists() or stamp.read_text().strip() != key:
            stale.append((name, key))
    if not stale:
        return found
    nvcc = _nvcc()
    _log(f"compiling {len(stale)} CUDA source{'s' if len(stale) > 1 else ''} for sm_100a into {build_dir} (first use only)", verbose)
    started = time.time()
    done = threading.Event()

    def heartbeat() -> None:
        while not done.wait(10.0):
            _log(f"still compiling ... {time.time() - started:.0f} s", verbose)

    def compile_one(item: tuple[str, str]) -> None:
        name, key = item
        made = build_dir / f"{found[name].name}.{os.getpid()}.tmp"
        try:
            cmd = [nvcc, *flags, "-shared", "-I", str(CSRC), str(known[name]), "-o", str(made)]
            result = subprocess.run(cmd, capture_output=True, text=True)
            if result.returncode != 0:
                raise BuildError(f"nvcc failed on {name}.cu:\n{result.stdout}\n{result.stderr}")
            os.replace(made, found[name])   # atomic: a concurrent process sees the old or the new file
            (build_dir / f"{name}{variant}.key").write_text(key)
        finally:
            made.unlink(missing_ok=True)
        _log(f"compiled {name}.cu ({time.time() - started:.0f} s)", verbose)

    threading.Thread(target=heartbeat, daemon=True).start()
    try:
        with ThreadPoolExecutor(max_workers=max(1, min(len(stale), os.cpu_count() or 1))) as pool:
            list(pool.map(compile_one, stale))
    finally:
        done.set()
    return found


if __name__ == "__main__":
    for path in library_paths(force="--force" in sys.argv).values():
        print(path)
