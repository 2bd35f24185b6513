"""Compiles libmgq.so in place when a fresh checkout does not have it yet (importing the package needs it)."""
import fcntl
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))


def ensure_library() -> None:
    target = os.path.join(HERE, "libmgq.so")
    if os.path.exists(target):
        return
    with open(os.path.join(HERE, ".build.lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)                      # one build, the others wait for it
        if os.path.exists(target):
            return
        env = dict(os.environ)
        if not any(os.access(os.path.join(p, "nvcc"), os.X_OK) for p in env.get("PATH", "").split(os.pathsep)):
            env["PATH"] = env.get("PATH", "") + os.pathsep + "/usr/local/cuda/bin"
        jobs = max(2, min(16, os.cpu_count() or 2))
        p = subprocess.run(["make", "-C", HERE, f"-j{jobs}", "libmgq.so"], env=env, stdin=subprocess.DEVNULL, stdout=subprocess.PIPE,
                           stderr=subprocess.STDOUT, text=True)
        if p.returncode:
            sys.stderr.write(p.stdout[-8000:])
            raise RuntimeError("compiling libmgq.so failed")
