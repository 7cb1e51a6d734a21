"""nvcc recipe for the library (sm_100a only, built in-tree).

``python tiny-gemma_b200/build.py [--force] [--verbose] [--family NAME]``

One translation unit per model family plus the common core, compiled in parallel into
``build/`` and linked into ``libtinygemma_b200.so``. ``--family`` builds the core and that
family alone (``libtinygemma_b200_<family>.so``): what a program that serves one model needs.
"""

from __future__ import annotations

import argparse
import fcntl
import os
import re
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "build")
LIB = os.path.join(HERE, "libtinygemma_b200.so")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
]
CORE = ["tg_core.cu"]
FAMILIES = {"gemma": ["tg_gemma.cu"], "hybrid": ["tg_hybrid.cu"]}


def lib_path(family: str | None = None) -> str:
    return LIB if family is None else LIB[:-3] + "_" + family + ".so"


def units(family: str | None = None) -> list[str]:
    fams = FAMILIES if family is None else {family: FAMILIES[family]}
    return CORE + [u for f in sorted(fams) for u in fams[f]]


def _deps(path: str, seen: set[str]) -> set[str]:
    """the file and the project headers it includes, transitively"""
    if path in seen or not os.path.exists(path):
        return seen
    seen.add(path)
    with open(path) as f:
        for inc in re.findall(r'^#include "([^"]+)"', f.read(), re.M):
            _deps(os.path.normpath(os.path.join(os.path.dirname(path), inc)), seen)
    return seen


def _newer(target: str, deps) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _unit_deps(unit: str) -> set[str]:
    return _deps(os.path.join(CSRC, unit), set())


def stale(family: str | None = None) -> bool:
    return any(_newer(lib_path(family), _unit_deps(u)) for u in units(family))


def build(force: bool = False, verbose: bool = False, family: str | None = None) -> str:
    lib = lib_path(family)
    if not force and not stale(family):
        return lib
    nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
    os.makedirs(OBJ, exist_ok=True)
    with open(os.path.join(OBJ, "lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)  # two processes may ask for the same library
        jobs = []
        for u in units(family):
            obj = os.path.join(OBJ, u[:-3] + ".o")
            if force or _newer(obj, _unit_deps(u)):
                cmd = [nvcc] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-c", "-o", obj + ".part", u]
                jobs.append((obj, cmd, subprocess.Popen(cmd, cwd=CSRC)))
        failed = None
        for obj, cmd, p in jobs:
            if p.wait() != 0:
                failed = subprocess.CalledProcessError(p.returncode, cmd)
            else:
                os.replace(obj + ".part", obj)
        if failed:
            raise failed
        objs = [os.path.join(OBJ, u[:-3] + ".o") for u in units(family)]
        subprocess.check_call([nvcc, "-gencode", "arch=compute_100a,code=sm_100a", "-shared", "-o", lib + ".part"] + objs, cwd=CSRC)
        os.replace(lib + ".part", lib)
    return lib


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--verbose", action="store_true")
    ap.add_argument("--family", choices=sorted(FAMILIES))
    a = ap.parse_args()
    print(build(a.force, a.verbose, a.family))
    sys.exit(0)
