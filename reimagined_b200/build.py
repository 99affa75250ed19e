"""In-tree build of the package's shared libraries for sm_100a with nvcc (no torch involvement).

    python -m reimagined_b200.build [ternary|stack ...] [--force] [--verbose]

libternary_b200.so holds the ternary linear path and the decode step of the hybrid that calls it;
libstack_b200.so the layer-stack models with dense weights.  Each is built from its own sources only, so a
process that serves one kind of model compiles nothing of the other.  The libraries land beside this file so
that they travel with the source tree.
"""
from __future__ import annotations

import fcntl
import hashlib
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIBRARIES = {
    "ternary": (os.path.join(HERE, "libternary_b200.so"),
                ["runtime.cu", "api.cu", "quantize.cu", "gemv_stream.cu", "gemv_generic.cu", "gemv_strip.cu",
                 "gemv_chain.cu", "gemm_tcgen05.cu", "gemm_widen.cu", "moe.cu", "glue.cu", "decode.cu", "packer.cpp",
                 "edge_pack.cpp"]),
    "stack": (os.path.join(HERE, "libstack_b200.so"),
              ["runtime.cu", "stack.cu", "stack_glue.cu", "dense.cu", "dense_rows.cu", "dense_tcgen05.cu", "delta_rule.cu",
               "latent_attention.cu", "latent_decode.cu", "latent_prefill.cu", "attention.cu", "attention_decode.cu",
               "attention_prefill.cu"]),
}
LIB, SOURCES = LIBRARIES["ternary"]
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
# IEEE division/sqrt and no fast-math: the fp32 epilogue and the quantiser scale are part of the
# bit-exact contract.  -lineinfo keeps profiler source correlation.
FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-O3", "-std=c++17", "-lineinfo",
         "--prec-div=true", "--prec-sqrt=true", "--fmad=true", "-Xcompiler", "-fPIC",
         "-Xptxas", "-v"]


def _digest(sources) -> str:
    """SHA-256 over the sources, the headers and the flags: what a library was built from."""
    h = hashlib.sha256(" ".join(FLAGS).encode())
    deps = [os.path.join(CSRC, f) for f in sorted(os.listdir(CSRC)) if f in sources or f.endswith(".cuh")]
    include = os.path.join(HERE, "..", "include")
    deps += [os.path.join(include, f) for f in sorted(os.listdir(include)) if f.endswith(".h")]
    for d in deps:
        h.update(os.path.basename(d).encode())
        with open(d, "rb") as f:
            h.update(f.read())
    return h.hexdigest()


def _stale(name: str) -> bool:
    # by content, not by time stamp: a copy of the tree (another machine, a fresh checkout) keeps the library valid
    lib, sources = LIBRARIES[name]
    if not os.path.exists(lib) or not os.path.exists(lib + ".sources"):
        return True
    with open(lib + ".sources") as f:
        return f.read().strip() != _digest(sources)


def build(force: bool = False, verbose: bool = False, libraries=tuple(LIBRARIES)) -> str:
    """Brings the named libraries up to date; returns the path of the first one."""
    stale = [n for n in libraries if force or _stale(n)]
    if stale:
        # one builder at a time: several ranks of one job may get here together
        os.makedirs(os.path.join(HERE, "build"), exist_ok=True)
        with open(os.path.join(HERE, "build", "lock"), "w") as lock:
            fcntl.flock(lock, fcntl.LOCK_EX)
            try:
                stale = [n for n in stale if force or _stale(n)]
                if stale:
                    _compile(stale, verbose)
            finally:
                fcntl.flock(lock, fcntl.LOCK_UN)
    return LIBRARIES[libraries[0]][0]


def _compile(names, verbose: bool) -> None:
    procs = []
    for src in sorted({s for n in names for s in LIBRARIES[n][1]}):
        cmd = [NVCC, *FLAGS, "-c", os.path.join(CSRC, src), "-o", os.path.join(HERE, "build", src + ".o")]
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    log = []
    failed = False
    for src, p in procs:
        out, _ = p.communicate()
        log.append(f"==== {src}\n{out}")
        failed |= p.returncode != 0
    with open(os.path.join(HERE, "build", "ptxas.log"), "w") as f:
        f.write("\n".join(log))
    if verbose or failed:
        print("\n".join(log))
    if failed:
        raise RuntimeError("nvcc failed; see output above")
    for name in names:
        lib, sources = LIBRARIES[name]
        # link beside the target and rename: a process that is loading the old library never sees a half-written file
        objs = [os.path.join(HERE, "build", s + ".o") for s in sources]
        subprocess.run([NVCC, "-shared", "-o", lib + ".tmp", *objs, "-lcudart"], check=True)
        os.replace(lib + ".tmp", lib)
        with open(lib + ".sources", "w") as f:
            f.write(_digest(sources))


if __name__ == "__main__":
    chosen = [a for a in sys.argv[1:] if not a.startswith("-")] or list(LIBRARIES)
    build(force="--force" in sys.argv, verbose="--verbose" in sys.argv, libraries=chosen)
    print("\n".join(LIBRARIES[n][0] for n in chosen))
