"""Builds the CUDA library in-tree with nvcc for sm_100a (cross-compiles without a GPU).

`build()` makes the whole library. `ensure(architecture)` is for a command that runs one model in a fresh checkout: it
returns the whole library if that is up to date, else a library of only the sources that model needs.

Every csrc/*.cu is compiled to an object under build/ (in parallel, only where the source or a header is newer than the
object) and the objects are linked into libtpx_b200.so beside this file. `TPX_DEBUG=1` in the environment adds
-DTPX_DEBUG, which compiles in the timing-experiment knobs and debug exports; the default build has none of them."""
import concurrent.futures
import fcntl
import glob
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
SO = os.path.join(HERE, "libtpx_b200.so")
OBJ_DIR = os.path.join(HERE, "build")
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
]


# sources of models that do not need the whole library (names without the tpx_ prefix)
COMPONENTS = {"Dofivik": ("api", "linear_bf16", "linear_f32", "postnorm", "latent", "latent_tc", "latent_dec", "delta"),
              "Vedizen": ("api", "linear_bf16", "linear_f32", "postnorm", "dyt", "gla", "diff", "diff_tc", "diff_dec")}


def sources():
    return sorted(glob.glob(os.path.join(HERE, "csrc", "*.cu")))


def _headers():
    return glob.glob(os.path.join(HERE, "csrc", "*.cuh")) + glob.glob(os.path.join(HERE, "..", "include", "*.h"))


def _flags():
    return NVCC_FLAGS + (["-DTPX_DEBUG"] if os.environ.get("TPX_DEBUG", "0") == "1" else [])


def _obj(src):
    tag = "dbg" if os.environ.get("TPX_DEBUG", "0") == "1" else "rel"
    return os.path.join(OBJ_DIR, os.path.basename(src)[:-3] + "." + tag + ".o")


def stale(so=SO, srcs=None):
    if not os.path.exists(so):
        return True
    t = os.path.getmtime(so)
    return any(os.path.getmtime(d) > t for d in (srcs or sources()) + _headers())


def build(force=False, verbose=False, so=SO, srcs=None):
    srcs = srcs or sources()
    if not force and not stale(so, srcs):
        return so
    nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
    os.makedirs(OBJ_DIR, exist_ok=True)
    hdr_t = max(os.path.getmtime(h) for h in _headers())
    todo = []
    for s in srcs:
        o = _obj(s)
        if force or not os.path.exists(o) or os.path.getmtime(o) < max(os.path.getmtime(s), hdr_t):
            todo.append((s, o))

    def compile_one(so):
        s, o = so
        cmd = [nvcc] + _flags() + (["-Xptxas", "-v"] if verbose else []) + ["-c", "-o", o, s]
        subprocess.check_call(cmd, stdout=sys.stderr)

    with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 1)) as ex:
        list(ex.map(compile_one, todo))
    part = so + f".{os.getpid()}"
    subprocess.check_call([nvcc, "-gencode", "arch=compute_100a,code=sm_100a", "-shared", "-o", part] + [_obj(s) for s in srcs])
    os.replace(part, so)
    return so


def ensure(architecture):
    """Path of an up-to-date library that serves the named architecture, built now if there is none."""
    if architecture not in COMPONENTS:
        return build()
    if not stale():
        return SO
    srcs = [os.path.join(HERE, "csrc", f"tpx_{n}.cu") for n in COMPONENTS[architecture]]
    so = os.path.join(HERE, f"libtpx_b200_{architecture.lower()}.so")
    with open(so + ".lock", "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return build(so=so, srcs=srcs)


if __name__ == "__main__":
    print(build(force=True, verbose=True))
