"""Build the in-tree CUDA extension for sm_100a.

`python -m miles_b200.ops.build` compiles every `.cu` / `.cpp` under `csrc/` with
`-gencode arch=compute_100a,code=sm_100a -lineinfo` into `miles_b200/ops/_build/miles_b200_C.so`.
nvcc cross-compiles without a GPU, so the build also runs on CPU-only machines; the resulting `.so`
stays in the tree (git-ignored) and is what `miles_b200.ops.cuda` loads at run time.
"""
from __future__ import annotations

import glob
import hashlib
import os

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
BUILD_DIR = os.path.join(HERE, "_build")
EXT_NAME = "miles_b200_C"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "--use_fast_math",
    "-U__CUDA_NO_HALF_OPERATORS__", "-U__CUDA_NO_BFLOAT16_OPERATORS__", "-U__CUDA_NO_HALF_CONVERSIONS__",
    "-U__CUDA_NO_BFLOAT16_CONVERSIONS__", "-U__CUDA_NO_HALF2_OPERATORS__", "-U__CUDA_NO_BFLOAT162_OPERATORS__",
]


def sources() -> list[str]:
    return sorted(glob.glob(os.path.join(CSRC, "*.cu")) + glob.glob(os.path.join(CSRC, "*.cpp")))


# What serving a layer-by-layer decoder (models/layered.py) takes: dense projections, sampling and the parts its layers need.  A
# checkout without a full build compiles only these (`build_serve`), into an extension of its own with the same interface.
SERVE_SUFFIX = "_serve"
SERVE_SOURCES = ["counter.cpp", "bindings.cpp", "bindings_more.cpp", "bindings_misc.cpp", "bindings_mixers.cpp", "gemm.cu", "gemm_small.cu",
                 "gemv.cu", "misc.cu", "mixers.cu", "paged_attend.cu"]
SERVE_PARTS = {
    "latent": ["attention_latent_tc.cu", "latent_attn.cu", "latent_decode.cu", "latent_decode_tc.cu"],
    "linear": ["linear_state.cu", "linear_chunk.cu"],
    "attention": ["attention_window_tc.cu", "window_decode.cu"],
    "prep": ["window_prep.cu"],
    "differential": ["diff_prep.cu"],
    "ssm": ["ssm_state.cu", "ssm_chunk.cu"],
    "delta": ["delta_state.cu", "delta_chunk.cu"],
    "experts": ["bindings_moe.cpp", "moe.cu", "experts_any.cu"],
}
_serving: str | None = None                   # the serving build this process asked for


def serve_kind(cfg) -> str:
    """Which serving build a layered configuration needs: the names of its parts."""
    from ..models.layered import AttentionSpec, DeltaSpec, DifferentialSpec, LatentSpec, LinearStateSpec, MoeSpec, SsmSpec

    of = {LatentSpec: {"latent"}, LinearStateSpec: {"linear"}, AttentionSpec: {"attention", "prep"}, DifferentialSpec: {"attention", "differential"},
          SsmSpec: {"ssm"}, DeltaSpec: {"delta"}}
    parts = set().union(*(of[type(s.mixer)] for s in cfg.layer_specs))
    if any(isinstance(s.mlp, MoeSpec) for s in cfg.layer_specs):
        parts.add("experts")
    return "_".join(sorted(parts))


def source_stamp() -> str:
    """Hash of every source, header and flag: what a built extension was made from."""
    h = hashlib.sha256(" ".join(NVCC_FLAGS).encode())
    for path in sorted(glob.glob(os.path.join(CSRC, "*"))):
        with open(path, "rb") as f:
            h.update(os.path.basename(path).encode() + b"\0" + f.read())
    return h.hexdigest()


def _is_current(so: str) -> bool:
    try:
        with open(so + ".stamp") as f:
            return os.path.exists(so) and f.read() == source_stamp()
    except OSError:
        return False


def _write_stamp(so: str):
    with open(so + ".stamp", "w") as f:
        f.write(source_stamp())


DEBUG_SUFFIX = "_debug"                       # the build with device-side index checks (csrc/debug.cuh)


def debug_requested() -> bool:
    return os.environ.get("MILES_DEBUG_KERNELS", "0") == "1"


def serve_so_path(kind: str) -> str:
    name = f"{SERVE_SUFFIX}_{kind}"
    return os.path.join(BUILD_DIR + name, EXT_NAME + name + ".so")


def build_serve(kind: str, verbose: bool = False) -> str:
    """Make sure an extension that can serve layer-by-layer decoders with these parts (`serve_kind`) is built from the sources as they are:
    an up-to-date full build if there is one, else the serving subset.  Returns its path; `load()` then picks the same one."""
    global _serving
    if _is_current(so_path(False)):
        return so_path(False)
    so = serve_so_path(kind)
    if not _is_current(so):
        from torch.utils import cpp_extension

        _toolchain_env()
        os.makedirs(os.path.dirname(so), exist_ok=True)
        parts = kind.split("_")
        cpp_extension.load(
            name=f"{EXT_NAME}{SERVE_SUFFIX}_{kind}", sources=[os.path.join(CSRC, f) for f in SERVE_SOURCES + sum((SERVE_PARTS[p] for p in parts), [])],
            extra_cflags=["-O3", "-std=c++17", "-DMB_SERVE_SUBSET", *(f"-DMB_SERVE_{p.upper()}" for p in parts)], extra_cuda_cflags=NVCC_FLAGS,
            extra_include_paths=[CSRC], build_directory=os.path.dirname(so), verbose=verbose, with_cuda=True)
        _write_stamp(so)
    _serving = kind
    return so


def _toolchain_env():
    # link against the system libstdc++.so (the same one libtorch uses); a toolchain that links it statically
    # gives the extension a second, uninitialised copy of the iostream state
    if os.path.exists("/usr/bin/g++"):
        os.environ["CXX"] = "/usr/bin/g++"
        os.environ["CC"] = "/usr/bin/gcc"
    os.environ.setdefault("MAX_JOBS", str(os.cpu_count() or 8))
    # torch adds its own -gencode list unless it finds one in the flags; ours targets sm_100a only
    os.environ.setdefault("TORCH_CUDA_ARCH_LIST", "10.0a")


def so_path(debug: bool | None = None) -> str:
    debug = debug_requested() if debug is None else debug
    return os.path.join(BUILD_DIR + (DEBUG_SUFFIX if debug else ""), EXT_NAME + (DEBUG_SUFFIX if debug else "") + ".so")


def build(verbose: bool = False, debug: bool = False):
    """Compile (incrementally, via ninja) and import the extension module.  `debug`: the variant whose kernels check the
    indices they take from tensors (`-DMILES_DEBUG_BOUNDS`; loaded instead of the normal one with MILES_DEBUG_KERNELS=1)."""
    from torch.utils import cpp_extension

    if debug:
        d = BUILD_DIR + DEBUG_SUFFIX
        os.makedirs(d, exist_ok=True)
        _toolchain_env()
        return cpp_extension.load(
            name=EXT_NAME + DEBUG_SUFFIX, sources=sources(), extra_cflags=["-O3", "-std=c++17"],
            extra_cuda_cflags=NVCC_FLAGS + ["-DMILES_DEBUG_BOUNDS"], extra_include_paths=[CSRC], build_directory=d, verbose=verbose,
            with_cuda=True, is_python_module=True)
    os.makedirs(BUILD_DIR, exist_ok=True)
    _toolchain_env()
    mod = cpp_extension.load(
        name=EXT_NAME, sources=sources(), extra_cflags=["-O3", "-std=c++17"], extra_cuda_cflags=NVCC_FLAGS,
        extra_include_paths=[CSRC], build_directory=BUILD_DIR, verbose=verbose, with_cuda=True)
    _write_stamp(so_path(False))
    return mod


def load():
    """Import the already-built extension from the tree (no compilation)."""
    import importlib.util

    import torch  # noqa: F401  (libtorch symbols must be loaded first)

    debug = debug_requested()
    path, suffix = so_path(debug), DEBUG_SUFFIX if debug else ""
    if not debug and not _is_current(path):
        built = sorted(glob.glob(BUILD_DIR + SERVE_SUFFIX + "_*"))
        for kind in [_serving] if _serving else [d[len(BUILD_DIR + SERVE_SUFFIX) + 1:] for d in built]:
            if _is_current(serve_so_path(kind)):
                path, suffix = serve_so_path(kind), f"{SERVE_SUFFIX}_{kind}"
                break
    if not os.path.exists(path):
        raise ImportError(
            f"{path} not found: build the CUDA extension with `python -m miles_b200.ops.build` "
            "(or `python -c 'import __graft_entry__ as g; g.build()'`)")
    spec = importlib.util.spec_from_file_location(EXT_NAME + suffix, path)
    mod = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(mod)
    return mod


if __name__ == "__main__":
    import sys

    m = build(verbose="-v" in sys.argv, debug="--debug" in sys.argv)
    print("built", so_path("--debug" in sys.argv), "with", len([n for n in dir(m) if not n.startswith("_")]), "entry points")
