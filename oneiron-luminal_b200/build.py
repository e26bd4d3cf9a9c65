"""Builds the library in place when it is missing or older than its sources (a fresh checkout's first run)."""
from __future__ import annotations

import fcntl
import os
import shutil
import subprocess

from .runtime import library_path

_CSRC = os.path.join(os.path.dirname(os.path.abspath(__file__)), "csrc")


def ensure_library() -> str:
    """Path of the library, after an up-to-date build; one process builds, others wait.  Raises when nothing can be built or loaded."""
    path = library_path()
    if shutil.which("make") is None or shutil.which(os.environ.get("NVCC", "nvcc")) is None:
        if not os.path.exists(path):
            raise RuntimeError("the library is not built, and make / nvcc are not available to build it")
        return path
    os.makedirs(os.path.join(_CSRC, "_obj"), exist_ok=True)
    with open(os.path.join(_CSRC, "_obj", ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        r = subprocess.run(["make", "-j", str(max(1, min(16, os.cpu_count() or 1)))], cwd=_CSRC, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    if r.returncode != 0:
        raise RuntimeError("building the library failed:\n" + r.stdout[-4000:])
    return path
