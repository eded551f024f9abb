"""Builds libns_b200.so in place when it is missing (csrc/Makefile, nvcc for sm_100a)."""
from __future__ import annotations

import fcntl
import os
import subprocess
import sys

from . import native

CSRC = os.path.join(os.path.dirname(os.path.abspath(__file__)), "csrc")


def make(jobs: int | None = None) -> None:
    env = dict(os.environ)
    env.setdefault("NVCC", "/usr/local/cuda/bin/nvcc")
    res = subprocess.run(["make", "-C", CSRC, f"-j{jobs or os.cpu_count() or 8}"], env=env, stdin=subprocess.DEVNULL, capture_output=True, text=True)
    if res.returncode != 0:
        sys.stderr.write(res.stdout[-4000:] + "\n" + res.stderr[-4000:])
        raise RuntimeError("building libns_b200.so failed")


def ensure() -> None:
    """The library exists afterwards; processes that start together build once."""
    if os.path.exists(native.LIB_PATH):
        return
    os.makedirs(os.path.join(CSRC, "build"), exist_ok=True)
    with open(os.path.join(CSRC, "build", ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not os.path.exists(native.LIB_PATH):
            make()
