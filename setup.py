"""Builds the sm_100a extension in-tree: `python setup.py build_ext --inplace`
produces fastcache_b200/_C*.so.  The arch flags are passed explicitly
(-gencode arch=compute_100a,code=sm_100a), which bypasses torch's own arch list;
nvcc cross-compiles without a GPU."""
import glob
import os

from setuptools import setup
from torch.utils.cpp_extension import BuildExtension, CUDAExtension

ROOT = os.path.dirname(os.path.abspath(__file__))
SRC = os.path.join("fastcache_b200", "csrc")
# FC_EXT=core: `fastcache_b200._C_core`, the part that models without per-head K/V attention, compression or tensor
# parallelism need (ops/loader.py takes it where the whole extension is not built)
CORE = os.environ.get("FC_EXT") == "core"
CORE_SOURCES = ("attn_decode.cu", "attn_prefill.cu", "attn_prefill_tc2.cu", "bindings.cpp", "elementwise.cu", "gemm.cu", "gemm_2cta.cu", "gemm_skinny.cu", "gemm_streamk.cu",
                "hybrid_bind.cpp", "latent.cu", "latent_decode.cu", "latent_decode_tc.cu", "latent_prefill.cu", "linear_simt.cu", "lru.cu", "moe.cu", "moe_gemm.cu", "partials.cu", "prenorm_bind.cpp",
                "recurrence.cu", "recurrence_chunk.cu", "resid.cu", "streams.cu", "streams_bind.cpp", "talking.cu", "talking_bind.cpp", "window_attn.cu")
sources = [os.path.join(SRC, f) for f in CORE_SOURCES] if CORE else sorted(glob.glob(os.path.join(SRC, "*.cu")) + glob.glob(os.path.join(SRC, "*.cpp")))

nvcc_flags = ["-O3", "-std=c++17", "-lineinfo", "-gencode", "arch=compute_100a,code=sm_100a",
              "--expt-relaxed-constexpr", "-Xptxas", "-v"] if os.environ.get("FC_PTXAS_V") else \
             ["-O3", "-std=c++17", "-lineinfo", "-gencode", "arch=compute_100a,code=sm_100a",
              "--expt-relaxed-constexpr"]

setup(
    name="fastcache_b200",
    version="0.1.0",
    packages=[],
    ext_modules=[CUDAExtension(
        name="fastcache_b200._C_core" if CORE else "fastcache_b200._C",
        sources=sources,
        include_dirs=[os.path.join(ROOT, SRC)],
        extra_compile_args={"cxx": ["-O3", "-std=c++17"], "nvcc": nvcc_flags},
    )],
    cmdclass={"build_ext": BuildExtension.with_options(use_ninja=True)},
)
