"""Build libmacllm_b200.so (sm_100a) in-tree with nvcc.

Usage: python macllm-infer_b200/build.py [--force]
Objects are cached under macllm-infer_b200/build/ and rebuilt when a source or header is newer.

build_for_serving() is what a fresh checkout needs to serve a safetensors checkpoint: the same library without the GGUF
formats, their quantised matmuls and the kernel-level entry points.  It compiles nothing when a current library is there.
"""
from __future__ import annotations

import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

HERE = Path(__file__).resolve().parent
CSRC = HERE / "csrc"
BUILD = HERE / "build"
LIB = HERE / "libmacllm_b200.so"
SERVING_LIB = HERE / "libmacllm_b200_serving.so"
# the translation units behind a safetensors checkpoint; the rest serves GGUF files and kernel-level callers
SERVING = ["attention.cu", "attention_tc.cu", "batch.cu", "channel_delta.cu", "c_api_core.cpp", "c_api_model.cpp", "device_lm.cpp", "embed.cu", "engine.cpp", "gated_scan.cu", "hgemm_tc.cu",
           "json.cpp", "kv_pool.cpp", "latent_attention.cu", "linear_state.cu", "mixer_lm.cpp", "mixer_lm_conv.cpp", "mixer_lm_output.cpp", "mixer_lm_side.cpp", "mixer_ops.cu", "mixer_spec.cpp", "mlstm.cu", "model_registry.cpp", "moe_rows.cu", "paged_lm.cpp",
           "rope_kv.cu", "safetensors_file.cpp", "sample.cu", "seed_model.cpp", "device_info.cpp", "weights.cpp"]

NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
COMMON = [
    "-std=c++17", "-O3", "-lineinfo",
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-Xcompiler", "-fPIC,-fopenmp,-Wall,-Wno-unknown-pragmas",
    "-I", str(HERE.parent / "include"),
]


def _newest_header() -> float:
    hs = list(CSRC.glob("*.h")) + list(CSRC.glob("*.cuh")) + list((HERE.parent / "include").glob("*.h"))
    return max(p.stat().st_mtime for p in hs)


def _stale(lib: Path, srcs) -> bool:
    return not lib.exists() or lib.stat().st_mtime < max(_newest_header(), max(p.stat().st_mtime for p in srcs))


def _all_sources():
    return sorted(list(CSRC.glob("*.cu")) + list(CSRC.glob("*.cpp")))


def _build(lib: Path, srcs, force: bool, verbose: bool) -> Path:
    BUILD.mkdir(exist_ok=True)
    hdr_time = _newest_header()
    jobs = []
    objs = []
    for s in srcs:
        o = BUILD / (s.name + ".o")
        objs.append(o)
        if force or not o.exists() or o.stat().st_mtime < max(s.stat().st_mtime, hdr_time):
            cmd = [NVCC, *COMMON, "-x", "cu", "-c", str(s), "-o", str(o)]
            if verbose:
                cmd.insert(1, "-Xptxas=-v")
            jobs.append(cmd)

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("nvcc failed:\n" + " ".join(cmd) + "\n" + r.stdout + r.stderr)
        return r.stderr

    if jobs:
        with ThreadPoolExecutor(max_workers=min(os.cpu_count() or 8, len(jobs))) as ex:
            for out in ex.map(run, jobs):
                if verbose and out:
                    print(out)
    if jobs or _stale(lib, objs):
        link = [NVCC, "-shared", "-o", str(lib), *map(str, objs), "-Xcompiler", "-fopenmp", "-lgomp", "-lcudart_static",
                "-gencode", "arch=compute_100a,code=sm_100a"]
        run(link)
    return lib


def build(force: bool = False, verbose: bool = False) -> Path:
    return _build(LIB, _all_sources(), force, verbose)


def build_for_serving() -> Path:
    if LIB.exists():
        return build()
    return _build(SERVING_LIB, [CSRC / n for n in SERVING], False, False)


if __name__ == "__main__":
    p = build(force="--force" in sys.argv, verbose="--verbose" in sys.argv)
    print(p)
