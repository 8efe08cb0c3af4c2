"""In-tree build of the native library: ``python -m vllm_ascend_b200.build``.

Every ``csrc/*.cu`` / ``csrc/*.cpp`` is compiled for sm_100a only and linked
into ``vllm_ascend_b200/_C.so`` (plain C ABI, loaded with ctypes by
``vllm_ascend_b200._native``).  Objects are cached by source hash so a rebuild
only recompiles what changed.  Build knobs follow the reference's env-driven
setup (setup.py:74-132): ``MAX_JOBS``, ``CMAKE_BUILD_TYPE``.
"""
from __future__ import annotations

import fcntl
import hashlib
import json
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ_DIR = os.path.join(HERE, "csrc", "build")
LIB_PATH = os.path.join(HERE, "_C.so")
MANIFEST = os.path.join(OBJ_DIR, "linked.json")

NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
ARCH_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a"]


def _common_flags() -> list[str]:
    debug = os.environ.get("CMAKE_BUILD_TYPE", "Release").lower() == "debug"
    flags = ["-std=c++17", "-lineinfo", "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=hidden",
             "--expt-relaxed-constexpr", "-I", CSRC]
    flags += ["-O0", "-g"] if debug else ["-O3"]      # index checks in the kernels are always on
    if os.environ.get("B200_PTXAS_VERBOSE"):
        flags += ["-Xptxas", "-v"]
    return flags


def _sources() -> list[str]:
    return sorted(os.path.join(CSRC, f) for f in os.listdir(CSRC)
                  if f.endswith((".cu", ".cpp")))


def _headers_digest() -> str:
    h = hashlib.sha256()
    for f in sorted(os.listdir(CSRC)):
        if f.endswith((".cuh", ".h", ".hpp")):
            with open(os.path.join(CSRC, f), "rb") as fh:
                h.update(fh.read())
    h.update(" ".join(f for f in _common_flags() if f != CSRC).encode())      # the same wherever the tree lies
    return h.hexdigest()


def _object_path(src: str, hdr_digest: str) -> str:
    with open(src, "rb") as fh:
        digest = hashlib.sha256(fh.read() + hdr_digest.encode()).hexdigest()[:16]
    return os.path.join(OBJ_DIR, f"{os.path.splitext(os.path.basename(src))[0]}.{digest}.o")


def _compile_one(src: str, hdr_digest: str, verbose: bool) -> tuple[str, bool]:
    base = os.path.splitext(os.path.basename(src))[0]
    obj = _object_path(src, hdr_digest)
    if os.path.exists(obj):
        return obj, False
    for old in os.listdir(OBJ_DIR):
        if old.startswith(base + ".") and old.endswith(".o"):
            os.remove(os.path.join(OBJ_DIR, old))
    part = f"{obj}.{os.getpid()}.part.o"        # an interrupted compilation leaves no object
    cmd = [NVCC, *ARCH_FLAGS, *_common_flags(), "-x", "cu", "-c", src, "-o", part]
    if verbose:
        print(" ".join(cmd), flush=True)
    res = subprocess.run(cmd, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError(f"nvcc failed for {src}:\n{res.stdout}\n{res.stderr}")
    os.replace(part, obj)
    if res.stderr.strip() and (verbose or os.environ.get("B200_PTXAS_VERBOSE")):
        print(res.stderr, file=sys.stderr)
    return obj, True


#: sources a model needs, for builds that compile no more than that (architecture -> names; others: all)
MODEL_SOURCES = {
    "Vofelix": ("activations", "attention_decode", "attention_mla_decode", "cache_ops", "gemm_bf16", "gemm_bf16_2cta",
                "latent_attention", "linear_attention", "mla_preprocess", "sampler", "stream_norm"),
    "Pegopel": ("activations", "attention_decode", "attention_decode_tc", "attention_tc", "attention_variant", "cache_ops",
                "gemm_bf16", "gemm_bf16_2cta", "qkv_prep", "sampler", "stream_norm"),
    "Dubizen": ("activations", "attention_decode", "attention_decode_tc", "attention_mla_decode", "attention_tc",
                "attention_variant", "cache_ops", "elementwise", "gemm_bf16", "gemm_bf16_2cta", "latent_attention",
                "mla_preprocess", "moe", "qkv_prep", "sampler", "stream_norm"),
    "Nevotar": ("activations", "attention_decode", "attention_decode_tc", "attention_tc", "attention_variant",
                "attention_wide", "cache_ops", "elementwise", "gemm_bf16", "gemm_bf16_2cta", "group_norm", "linear_attention",
                "linear_recurrence", "moe", "qkv_prep", "sampler", "stream_norm"),
}


def _linked() -> list[str]:
    """Names of the objects in the present library ([]: unknown)."""
    try:
        with open(MANIFEST) as fh:
            return json.load(fh) if os.path.exists(LIB_PATH) else []
    except (OSError, ValueError):
        return []


def build(verbose: bool = False, force: bool = False, sources=None) -> str:
    """Compile and link the native library; returns its path.  ``sources`` (names without suffix)
    limits the compilation to these files and what a present library holds already; a later call
    without the limit adds the rest."""
    os.makedirs(OBJ_DIR, exist_ok=True)
    with open(os.path.join(OBJ_DIR, ".lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return _build_locked(verbose, force, sources)


def _build_locked(verbose: bool, force: bool, sources) -> str:
    if force:
        for f in os.listdir(OBJ_DIR):
            if f != ".lock":
                os.remove(os.path.join(OBJ_DIR, f))
    hdr = _headers_digest()
    srcs = _sources()
    if sources is not None:
        names = set(sources)
        known = {os.path.splitext(os.path.basename(s))[0] for s in srcs}
        if names - known:
            raise ValueError(f"no such source: {sorted(names - known)}")
        if os.path.exists(LIB_PATH):        # never shrink a library: what it holds is kept up to date as well
            held = {o.split(".")[0] for o in _linked()}
            names = names | held if held else known
        wanted = [s for s in srcs if os.path.splitext(os.path.basename(s))[0] in names]
    else:
        wanted = srcs
    jobs = int(os.environ.get("MAX_JOBS", os.cpu_count() or 4))
    with ThreadPoolExecutor(max_workers=jobs) as ex:
        results = list(ex.map(lambda s: _compile_one(s, hdr, verbose), wanted))
    objs = [o for o, _ in results]
    linked = _linked()
    if set(map(os.path.basename, objs)) <= set(linked):
        return LIB_PATH
    objs += [o for o in (_object_path(s, hdr) for s in srcs if s not in wanted) if os.path.exists(o)]
    # linked under another name first: a library that is loaded somewhere is replaced, not written over
    tmp = f"{LIB_PATH}.{os.getpid()}.tmp"
    cmd = [NVCC, *ARCH_FLAGS, "-shared", "-o", tmp, *objs,
           "-cudart", "static", "-Xlinker", "--no-undefined", "-lpthread", "-ldl", "-lrt"]
    if verbose:
        print(" ".join(cmd), flush=True)
    res = subprocess.run(cmd, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError(f"link failed:\n{res.stdout}\n{res.stderr}")
    os.replace(tmp, LIB_PATH)
    with open(MANIFEST, "w") as fh:
        json.dump(sorted(map(os.path.basename, objs)), fh)
    return LIB_PATH


def ensure(architecture: str) -> str:
    """Library with everything ``architecture`` needs, compiled from the present sources."""
    return build(sources=MODEL_SOURCES.get(architecture))


if __name__ == "__main__":
    path = build(verbose="-v" in sys.argv, force="--force" in sys.argv)
    print(path)
