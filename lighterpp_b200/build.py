"""Compiles the CUDA library from the sources beside it when it is not there yet (a fresh checkout)."""
from __future__ import annotations

import fcntl
import os
import subprocess

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "liblpp_b200.so")


def ensure_built() -> str:
    """Path of the library; builds it (one or two minutes) when it is missing.  Callers that race for it wait for the one
    that builds, and the finished library appears under its name in one step."""
    if os.path.exists(LIB_PATH):
        return LIB_PATH
    with open(LIB_PATH + ".lock", "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not os.path.exists(LIB_PATH):
            part = f"{LIB_PATH}.{os.getpid()}.part"
            env = dict(os.environ, LPP_OUT=part)
            r = subprocess.run(["sh", os.path.join(_HERE, "csrc", "build.sh")], env=env, stdin=subprocess.DEVNULL, capture_output=True, text=True)
            if r.returncode != 0:
                raise RuntimeError("nvcc build failed:\n" + r.stdout[-2000:] + r.stderr[-4000:])
            os.replace(part, LIB_PATH)
    return LIB_PATH
