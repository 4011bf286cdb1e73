"""Builds libtsb.so (the C-ABI shared library) in-tree with nvcc for sm_100a.

    python -m turbospark_b200.build [--force] [--verbose]

Every .cu under csrc/ is compiled to an object under _build/ (only when stale)
and linked into turbospark_b200/libtsb.so.  No CPU fallback exists: if this
library is missing the package refuses to load.
"""
import concurrent.futures
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
# TSB_BUILD_DIR redirects objects and the library (a scratch build that leaves the in-tree library alone)
OUT = os.path.join(os.environ["TSB_BUILD_DIR"], "obj") if os.environ.get("TSB_BUILD_DIR") else os.path.join(HERE, "_build")
LIB = os.path.join(os.environ["TSB_BUILD_DIR"], "libtsb.so") if os.environ.get("TSB_BUILD_DIR") else os.path.join(HERE, "libtsb.so")
INCLUDE = os.path.join(os.path.dirname(HERE), "include")

NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC,-fvisibility=hidden,-Wall", "--expt-relaxed-constexpr",
    "-I", INCLUDE,
] + os.environ.get("TSB_NVCC_EXTRA", "").split()


# Units of one model family only; a library of one family leaves the other's out (build(family=...)).
FAMILY_UNITS = {
    "blocks": {"attention.cu", "attention_tc.cu", "comm.cu", "gemm_quant.cu", "gemm_wide.cu", "model_blocks.cu", "moe.cu", "resident.cu", "rowops.cu"},
    "plain": {"attention_kv.cu", "attention_kv_tc.cu", "attention_latent.cu", "attention_prefix.cu", "attention_prefix_tc.cu", "attention_window.cu", "attention_window_tc.cu", "experts.cu", "gemm_plain.cu",
              "model_plain.cu", "ops_plain.cu", "recurrence.cu", "recurrence_chunks.cu", "rowops_plain.cu", "scan.cu", "sublayer.cu"},
}


def _sources(family=None):
    other = set().union(*(u for f, u in FAMILY_UNITS.items() if f != family)) if family else set()
    return sorted(f for f in os.listdir(CSRC) if f.endswith(".cu") and f not in other)


def _stale(out, deps):
    return not os.path.exists(out) or os.path.getmtime(out) < max(os.path.getmtime(d) for d in deps)


def _headers_mtime():
    hs = [os.path.join(CSRC, f) for f in os.listdir(CSRC) if f.endswith((".cuh", ".h"))]
    hs.append(os.path.join(INCLUDE, "tsb.h"))
    return max(os.path.getmtime(h) for h in hs)


def _compile(src, verbose):
    obj = os.path.join(OUT, src[:-3] + ".o")
    cmd = [NVCC] + FLAGS + (["-Xptxas", "-v"] if verbose else []) + ["-c", os.path.join(CSRC, src), "-o", obj]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError("nvcc failed for %s:\n%s\n%s" % (src, r.stdout, r.stderr))
    return src, r.stderr


def build(force=False, verbose=False, family=None):
    """Compile what is stale and link.  family: only that model family's units and the common ones, into a library of its
    own; None: everything, into libtsb.so.  Returns the library's path."""
    os.makedirs(OUT, exist_ok=True)
    lib = LIB if family is None else LIB[:-3] + "_%s.so" % family
    hm = _headers_mtime()
    todo, objs = [], []
    for src in _sources(family):
        obj = os.path.join(OUT, src[:-3] + ".o")
        objs.append(obj)
        stale = (force or not os.path.exists(obj)
                 or os.path.getmtime(obj) < max(os.path.getmtime(os.path.join(CSRC, src)), hm))
        if stale:
            todo.append(src)
    logs = []
    if todo:
        with concurrent.futures.ThreadPoolExecutor(max_workers=min(8, len(todo))) as ex:
            for src, log in ex.map(lambda s: _compile(s, verbose), todo):
                logs.append((src, log))
    if todo or _stale(lib, objs):
        part = "%s.%d" % (lib, os.getpid())
        cmd = [NVCC, "-shared", "-o", part] + objs + ["-gencode", "arch=compute_100a,code=sm_100a", "-lcudart"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("link failed:\n%s\n%s" % (r.stdout, r.stderr))
        os.replace(part, lib)
    if verbose:
        for src, log in logs:
            print("==", src)
            print(log)
    return lib


def ensure(family):
    """A library that serves models of this family: the full one when it is newer than every source, else the family's own,
    compiled as far as needed."""
    deps = [os.path.join(CSRC, f) for f in os.listdir(CSRC)] + [os.path.join(INCLUDE, "tsb.h")]
    return LIB if not _stale(LIB, deps) else build(family=family)


if __name__ == "__main__":
    build(force="--force" in sys.argv, verbose="--verbose" in sys.argv)
    print(LIB)
