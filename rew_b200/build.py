"""Builds librew_b200.so (CUDA, sm_100a only) in-tree with nvcc.

Usage: python -m rew_b200.build [--force]
"""
import concurrent.futures
import fcntl
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OUT = os.path.join(HERE, "librew_b200.so")
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC,-fvisibility=hidden", "--expt-relaxed-constexpr",
    "-I", os.path.join(HERE, "..", "include"), "-I", "/usr/include",
]


def sources():
    return sorted(f for f in os.listdir(CSRC) if f.endswith(".cu"))


def _stale(target, deps):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _compile(src, verbose):
    obj = os.path.join(CSRC, src[:-3] + ".o")
    headers = [os.path.join(CSRC, h) for h in os.listdir(CSRC) if h.endswith(".cuh")]
    headers.append(os.path.join(HERE, "..", "include", "rew_b200.h"))
    if _stale(obj, [os.path.join(CSRC, src)] + headers):
        cmd = [NVCC] + FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-c", os.path.join(CSRC, src), "-o", obj]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("nvcc failed for %s:\n%s\n%s" % (src, r.stdout, r.stderr))
        return obj, r.stderr
    return obj, ""


def build(force=False, verbose=False):
    """Compiles what is missing or out of date; processes that start together wait for one another."""
    with open(os.path.join(HERE, ".build.lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return _build(force, verbose)


def _build(force, verbose):
    srcs = sources()
    if force:
        for s in srcs:
            o = os.path.join(CSRC, s[:-3] + ".o")
            if os.path.exists(o):
                os.remove(o)
    with concurrent.futures.ThreadPoolExecutor(max_workers=os.cpu_count() or 4) as ex:
        results = list(ex.map(lambda s: _compile(s, verbose), srcs))
    objs = [o for o, _ in results]
    log = "".join(l for _, l in results)
    if _stale(OUT, objs):
        part = OUT + ".part"
        cmd = [NVCC, "-shared", "-o", part] + objs + ["-gencode", "arch=compute_100a,code=sm_100a", "-ldl"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("link failed:\n%s\n%s" % (r.stdout, r.stderr))
        os.replace(part, OUT)
    return OUT, log


if __name__ == "__main__":
    out, log = build(force="--force" in sys.argv, verbose="-v" in sys.argv)
    if log:
        print(log)
    print(out)
