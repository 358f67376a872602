"""Build recipe of the CUDA library (stands in for the reference's build.rs, which compiles its
kernels with nvcc at build time).  Produces ``liblfm25_b200.so`` next to this file, for sm_100a only.

    python lfm25-inference_b200/build.py [--force] [--verbose]

Every source is compiled to an object of its own (in parallel, only when it or a header changed) under
``build/`` and the objects are linked into the shared library.  A digest of the sources beside the library tells
whether it is up to date where the objects were not kept.  ``--verbose`` adds ``-Xptxas -v``.
"""
from __future__ import annotations

import hashlib
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJECTS = os.path.join(HERE, "build")
OUTPUT = os.path.join(HERE, "liblfm25_b200.so")
DIGEST = OUTPUT + ".sources"
SOURCES = ["api.cu", "options.cu", "attention.cu", "kv_cache.cu", "fp8_elementwise.cu", "fp8_gemm_stream.cu",
           "fp8_gemm_umma.cu", "gemm_rows_umma.cu", "attention_static_scratch.cu", "hybrid_attention.cu",
           "hybrid_attention_umma.cu", "model_ops.cu", "cublaslt_bf16.cu", "decode_executor.cu", "host_runtime.cu",
           "prefix_cache.cu", "scheduler.cu", "serving_engine.cu", "step_backends.cu", "stack_norm.cu", "stack_attention.cu",
           "stack_attention_umma.cu", "stack_attention_decode.cu", "delta_rule.cu", "head_linear.cu", "stack_latent.cu",
           "stack_latent_decode.cu", "state_space.cu", "state_space_chunk.cu", "stack_executor.cu"]
COMPILE_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC"]
LINK_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-shared", "-cudart", "static", "-ldl"]


def _headers() -> list[str]:
    found = [os.path.join(CSRC, name) for name in os.listdir(CSRC) if name.endswith((".h", ".cuh"))]
    found.append(os.path.join(HERE, "..", "include", "lfm25_b200.h"))
    found.append(os.path.abspath(__file__))
    return found


def _digest() -> str:
    digest = hashlib.sha256()
    for path in sorted([os.path.join(CSRC, name) for name in SOURCES] + _headers()):
        with open(path, "rb") as handle:
            digest.update(os.path.basename(path).encode() + b"\0" + hashlib.sha256(handle.read()).digest())
    return digest.hexdigest()


def _up_to_date(digest: str) -> bool:
    if not (os.path.exists(OUTPUT) and os.path.exists(DIGEST)):
        return False
    with open(DIGEST) as handle:
        return handle.read().strip() == digest


def _newer_than(target: str, inputs: list[str]) -> bool:
    if not os.path.exists(target):
        return True
    built = os.path.getmtime(target)
    return any(os.path.getmtime(path) > built for path in inputs)


def _compile(nvcc: str, source: str, obj: str, verbose: bool) -> tuple[int, str]:
    flags = COMPILE_FLAGS + (["-Xptxas", "-v"] if verbose else [])
    result = subprocess.run([nvcc, *flags, "-c", source, "-o", obj], capture_output=True, text=True)
    return result.returncode, result.stdout + result.stderr


def build(force: bool = False, verbose: bool = False) -> str:
    digest = _digest()
    if not force and _up_to_date(digest):
        return OUTPUT
    nvcc = os.environ.get("NVCC", "nvcc")
    os.makedirs(OBJECTS, exist_ok=True)
    headers = _headers()
    jobs = []
    objects = []
    for name in SOURCES:
        source = os.path.join(CSRC, name)
        obj = os.path.join(OBJECTS, name[:-3] + ".o")
        objects.append(obj)
        if force or _newer_than(obj, [source, *headers]):
            jobs.append((source, obj))
    failed = False
    with ThreadPoolExecutor(max_workers=min(8, os.cpu_count() or 1)) as pool:
        for code, output in pool.map(lambda job: _compile(nvcc, job[0], job[1], verbose), jobs):
            if verbose or code != 0:
                sys.stderr.write(output)
            failed = failed or code != 0
    if failed:
        raise RuntimeError("nvcc failed compiling the library sources")
    if jobs or force or _newer_than(OUTPUT, objects):
        result = subprocess.run([nvcc, *LINK_FLAGS, "-o", OUTPUT, *objects], capture_output=True, text=True)
        if verbose or result.returncode != 0:
            sys.stderr.write(result.stdout + result.stderr)
        if result.returncode != 0:
            raise RuntimeError(f"nvcc failed linking {os.path.basename(OUTPUT)}")
    with open(DIGEST, "w") as handle:
        handle.write(digest + "\n")
    return OUTPUT


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="--verbose" in sys.argv))
