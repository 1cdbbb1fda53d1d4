"""In-tree build of the native libraries (``python -m rumus_b200.build``).

* every ``csrc/kernels/*.cu`` and ``csrc/comm/*.cu`` is compiled for sm_100a only
  (``-gencode arch=compute_100a,code=sm_100a``) and linked into
  ``rumus_b200/lib/librumus_b200_cuda.so``;
* every ``csrc/{cpu_oracle,serve,runtime}/*.cpp`` is compiled with g++ into
  ``rumus_b200/lib/librumus_b200_host.so``.

``python -m rumus_b200.build --part NAME`` builds only what one family of models needs (``PARTS``).

Objects are cached under ``build/obj`` keyed by source + header mtimes, libraries by the content of their
sources, and translation units compile in parallel.  nvcc cross-compiles, so this runs on a
machine without a GPU.
"""
from __future__ import annotations

import concurrent.futures as cf
import glob
import hashlib
import os
import shutil
import subprocess
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CSRC = os.path.join(ROOT, "csrc")
OBJ = os.path.join(ROOT, "build", "obj")
LIB = os.path.join(ROOT, "rumus_b200", "lib")

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=default",
    "--expt-relaxed-constexpr",
]
CXX_FLAGS = ["-O2", "-std=c++17", "-fPIC", "-pthread", "-Wall"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found")


# Parts: a subset of the sources that one family of models needs, linked into libraries of their own
# (``librumus_b200_{cuda,host}_<part>.so``) so that serving such a model from a fresh checkout does not
# wait for kernels it never launches.
PARTS = {
    "latent": (["runtime.cu", "gemm.cu", "gemm_bf16.cu", "gemm_2cta.cu", "gemm_rows.cu", "elementwise.cu", "paged_attention.cu",
                "residual_stream.cu", "latent_attention.cu", "latent_decode.cu", "latent_prefill.cu"],
               ["kv_scheduler.cpp"]),
    "window": (["runtime.cu", "gemm.cu", "gemm_bf16.cu", "gemm_2cta.cu", "gemm_rows.cu", "elementwise.cu", "paged_attention.cu",
                "residual_stream.cu", "latent_attention.cu", "window_attention.cu", "window_decode.cu",
                "window_prefill.cu", "moe.cu", "moe_gemm.cu"],
               ["kv_scheduler.cpp"]),
    "hybrid": (["runtime.cu", "gemm.cu", "gemm_bf16.cu", "gemm_2cta.cu", "gemm_rows.cu", "elementwise.cu", "paged_attention.cu",
                "residual_stream.cu", "latent_attention.cu", "window_attention.cu", "window_decode.cu",
                "window_prefill.cu", "moe.cu", "moe_gemm.cu", "recurrent.cu", "mlstm_chunk.cu",
                "delta_chunk.cu"],
               ["kv_scheduler.cpp"]),
    "talk": (["runtime.cu", "gemm.cu", "gemm_bf16.cu", "gemm_2cta.cu", "gemm_rows.cu", "elementwise.cu", "paged_attention.cu",
              "residual_stream.cu", "latent_attention.cu", "talk_attention.cu", "talk_decode.cu", "talk_prefill.cu", "recurrent.cu", "delta_chunk.cu"],
             ["kv_scheduler.cpp"]),
}


def _headers_stamp(dirs) -> str:
    h = hashlib.sha1()
    for d in dirs:
        for f in sorted(glob.glob(os.path.join(d, "*.cuh")) + glob.glob(os.path.join(d, "*.h"))
                        + glob.glob(os.path.join(d, "*.hpp"))):
            h.update(os.path.relpath(f, ROOT).encode())
            h.update(str(os.path.getmtime(f)).encode())
    return h.hexdigest()[:12]


def _digest(srcs, dirs, flags) -> str:
    """Content hash of a library's sources, the headers next to them and the flags; it lies beside the
    library, so a library that was built elsewhere from the same files counts as current."""
    h = hashlib.sha1(" ".join(flags).encode())
    heads = sum((glob.glob(os.path.join(d, "*" + e)) for d in dirs for e in (".cuh", ".h", ".hpp")), [])
    for f in sorted(srcs) + sorted(heads):
        h.update(os.path.relpath(f, ROOT).encode())
        with open(f, "rb") as fh:
            h.update(fh.read())
    return h.hexdigest()


def library_current(so: str, digest: str) -> bool:
    try:
        with open(so + ".digest") as f:
            return os.path.exists(so) and f.read() == digest
    except OSError:
        return False


def _sources(part=None):
    cu_dirs = [os.path.join(CSRC, "kernels"), os.path.join(CSRC, "comm")]
    cpp_dirs = [os.path.join(CSRC, d) for d in ("cpu_oracle", "serve", "runtime")]
    cu = sorted(sum((glob.glob(os.path.join(d, "*.cu")) for d in cu_dirs), []))
    cpp = sorted(sum((glob.glob(os.path.join(d, "*.cpp")) for d in cpp_dirs), []))
    if part is not None:
        cu = [f for f in cu if os.path.basename(f) in PARTS[part][0]]
        cpp = [f for f in cpp if os.path.basename(f) in PARTS[part][1]]
    return cu_dirs, cpp_dirs, cu, cpp


def lib_paths(part=None):
    tail = f"_{part}.so" if part else ".so"
    return os.path.join(LIB, "librumus_b200_cuda" + tail), os.path.join(LIB, "librumus_b200_host" + tail)


def ensure(part: str | None) -> str | None:
    """Makes the libraries for ``part`` available: the complete ones when they are current, else the
    part's own, compiled if need be.  Returns the part to load (None = the complete libraries)."""
    cu_dirs, cpp_dirs, cu, cpp = _sources()
    cuda_so, host_so = lib_paths()
    if library_current(cuda_so, _digest(cu, cu_dirs, NVCC_FLAGS)) and \
            library_current(host_so, _digest(cpp, cpp_dirs, CXX_FLAGS)):
        return None
    build(part=part)
    return part


def _compile(cmd, out, stamp_file, stamp):
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError("compile failed: " + " ".join(cmd) + "\n" + r.stdout + r.stderr)
    with open(stamp_file, "w") as f:
        f.write(stamp)
    return out, r.stderr


def build(verbose: bool = False, jobs: int | None = None, part: str | None = None) -> dict:
    os.makedirs(OBJ, exist_ok=True)
    os.makedirs(LIB, exist_ok=True)
    cu_dirs, cpp_dirs, cu_srcs, cpp_srcs = _sources(part)
    cuda_so, host_so = lib_paths(part)
    cu_digest, cpp_digest = _digest(cu_srcs, cu_dirs, NVCC_FLAGS), _digest(cpp_srcs, cpp_dirs, CXX_FLAGS)
    info = {"compiled": 0, "cuda_so": cuda_so, "host_so": host_so, "cu_sources": len(cu_srcs),
            "cpp_sources": len(cpp_srcs)}
    if not verbose and library_current(cuda_so, cu_digest) and library_current(host_so, cpp_digest):
        return info
    nvcc = _nvcc()
    hstamp_cu = _headers_stamp(cu_dirs)
    hstamp_cpp = _headers_stamp(cpp_dirs)
    inc = sum((["-I", d] for d in cu_dirs + cpp_dirs), [])
    extra = ["-Xptxas", "-v"] if verbose else []

    tasks = []
    cu_objs, cpp_objs = [], []
    for src in cu_srcs:
        obj = os.path.join(OBJ, os.path.basename(src) + ".o")
        cu_objs.append(obj)
        stamp = f"{os.path.getmtime(src)}:{hstamp_cu}:{' '.join(NVCC_FLAGS)}"
        sf = obj + ".stamp"
        if os.path.exists(obj) and os.path.exists(sf) and open(sf).read() == stamp:
            continue
        tasks.append(([nvcc] + NVCC_FLAGS + extra + inc + ["-c", src, "-o", obj], obj, sf, stamp))
    for src in cpp_srcs:
        obj = os.path.join(OBJ, os.path.basename(src) + ".o")
        cpp_objs.append(obj)
        stamp = f"{os.path.getmtime(src)}:{hstamp_cpp}:{' '.join(CXX_FLAGS)}"
        sf = obj + ".stamp"
        if os.path.exists(obj) and os.path.exists(sf) and open(sf).read() == stamp:
            continue
        tasks.append((["g++"] + CXX_FLAGS + inc + ["-c", src, "-o", obj], obj, sf, stamp))

    jobs = jobs or max(1, (os.cpu_count() or 4))
    logs = []
    with cf.ThreadPoolExecutor(max_workers=jobs) as ex:
        futs = [ex.submit(_compile, *t) for t in tasks]
        for f in futs:
            out, log = f.result()
            if verbose and log:
                logs.append(log)
    for so, digest, cmd in (
            (cuda_so, cu_digest, [nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o"]),
            (host_so, cpp_digest, ["g++", "-shared", "-pthread", "-o"])):
        if library_current(so, digest):
            continue
        tmp = f"{so}.{os.getpid()}.tmp"
        r = subprocess.run(cmd + [tmp] + (cu_objs if so == cuda_so else cpp_objs), capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("link failed:\n" + r.stdout + r.stderr)
        os.replace(tmp, so)
        with open(so + ".digest", "w") as f:
            f.write(digest)
    if verbose:
        for l in logs:
            sys.stderr.write(l)
    info["compiled"] = len(tasks)
    return info


if __name__ == "__main__":
    part = sys.argv[sys.argv.index("--part") + 1] if "--part" in sys.argv else None
    info = build(verbose="-v" in sys.argv, part=part)
    print(info)
