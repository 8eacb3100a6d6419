"""Build vx_b200/libvx_cuda_dispatch.so from csrc/*.cu with nvcc for sm_100a.

for_parallel_decoders() and for_stream_decoders() give a library that can serve one
kind of decoder (of parallel blocks; of several residual streams): the whole one where
it is built and up to date, else a smaller one of the same objects,
libvx_parallel_decoder.so or libvx_stream_decoder.so, which takes less compiling.

The library is built in-tree, so that it travels with the source directory; it
links the CUDA runtime statically and opens libcuda.so.1 and libnccl.so.2 at
run time, so it loads (and answers symbol queries) on a machine with no GPU.
"""
import concurrent.futures
import os
import shutil
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "_obj")
LIB = os.path.join(HERE, "libvx_cuda_dispatch.so")
PARALLEL_LIB = os.path.join(HERE, "libvx_parallel_decoder.so")
STREAM_LIB = os.path.join(HERE, "libvx_stream_decoder.so")
NVCC = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"

SOURCES = ["rowdot_quant.cu", "rowdot_bf16.cu", "rowdot_f32.cu", "nn_kernels.cu",
           "dispatch.cu", "gemm_simt.cu", "gemm_umma.cu", "gemm_umma_pair.cu",
           "nn_api.cu", "decoder.cu", "decoder_parallel.cu", "flash_attn.cu",
           "flash_attn_v2.cu", "static_scratch.cu", "rowdot_umma.cu", "prefill.cu",
           "quantize.cu", "step_kernel.cu", "gemm_f32_split.cu", "moe_group.cu",
           "moe_grouped.cu", "gemm_fp8_rows.cu", "window_attention.cu",
           "parallel_block.cu", "tensor_map.cu", "decoder_streams.cu",
           "latent_attention.cu", "gated_linear.cu", "residual_streams.cu",
           "rowdot_streams_bf16.cu", "rowdot_streams_f32.cu"]
# what the decoders run and load their weights with; absent*.cu stand for the rest
_DECODER_SOURCES = ["nn_kernels.cu", "dispatch.cu", "nn_api.cu", "decoder.cu",
                    "prefill.cu", "parallel_block.cu", "tensor_map.cu", "absent.cu"]
PARALLEL_SOURCES = _DECODER_SOURCES + [
    "rowdot_bf16.cu", "rowdot_f32.cu", "decoder_parallel.cu", "window_attention.cu",
    "absent_streams.cu"]
STREAM_SOURCES = _DECODER_SOURCES + [
    "rowdot_streams_bf16.cu", "rowdot_streams_f32.cu", "decoder_streams.cu",
    "latent_attention.cu", "gated_linear.cu", "residual_streams.cu",
    "absent_parallel.cu"]
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3",
              "-std=c++17", "-Xcompiler", "-fPIC", "-Xcompiler", "-Wall",
              "-I" + os.path.join(ROOT, "include"),
              "-I" + os.path.join(HERE, "runtime"), "-I" + CSRC]


def _newer_than(target, deps):
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def _headers():
    out = []
    for d in (CSRC, os.path.join(HERE, "runtime"), os.path.join(ROOT, "include")):
        out += [os.path.join(d, f) for f in os.listdir(d)
                if f.endswith((".h", ".cuh"))]
    return out


def _compile(src, verbose):
    obj = os.path.join(OBJ, src.replace(".cu", ".o"))
    path = os.path.join(CSRC, src)
    if not _newer_than(obj, [path] + _headers()):
        return obj, ""
    cmd = [NVCC] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + \
          ["-c", path, "-o", obj]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError("nvcc failed on %s:\n%s" % (src, r.stderr))
    return obj, r.stderr


def _up_to_date(lib, sources):
    return not _newer_than(lib, [os.path.join(CSRC, f) for f in sources] + _headers())


def _library(lib, sources, verbose=False):
    with concurrent.futures.ThreadPoolExecutor(max_workers=8) as pool:
        results = list(pool.map(lambda s: _compile(s, verbose), sources))
    objs = [o for o, _ in results]
    if verbose:
        for _, log in results:
            sys.stderr.write(log)
    if _newer_than(lib, objs):
        cmd = [NVCC, "-shared", "-gencode", "arch=compute_100a,code=sm_100a",
               "-o", lib + ".tmp"] + objs + ["-ldl", "-lpthread",
                                             "-Xlinker", "--no-undefined"]
        subprocess.run(cmd, check=True)
        os.replace(lib + ".tmp", lib)
    return lib


def build(force=False, verbose=False):
    os.makedirs(OBJ, exist_ok=True)
    if force:
        for f in os.listdir(OBJ):
            os.remove(os.path.join(OBJ, f))
    return _library(LIB, SOURCES, verbose)


def _whole_or(lib, sources):
    if os.path.exists(LIB) and _up_to_date(LIB, SOURCES):
        return LIB
    os.makedirs(OBJ, exist_ok=True)
    return _library(lib, sources)


def for_parallel_decoders():
    return _whole_or(PARALLEL_LIB, PARALLEL_SOURCES)


def for_stream_decoders():
    return _whole_or(STREAM_LIB, STREAM_SOURCES)


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
