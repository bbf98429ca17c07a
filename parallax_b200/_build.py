"""In-tree build of the sm_100a kernel library (``parallax_b200/_C/libpxl_kernels.so``).

The kernel sources under ``csrc/`` expose a C ABI and include no PyTorch headers, so each
translation unit compiles in a few seconds with plain ``nvcc``; the Python side binds the
symbols with ``ctypes``. The library is kept inside the package directory so that a source
checkout carries its own binaries from the build machine to the GPU machine.
"""

from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

REPO_ROOT = Path(__file__).resolve().parent.parent
CSRC = REPO_ROOT / "csrc"
OUT_DIR = Path(__file__).resolve().parent / "_C"
LIB_NAME = "libpxl_kernels.so"

NVCC_FLAGS = [
    "-gencode",
    "arch=compute_100a,code=sm_100a",
    "-lineinfo",
    "-O3",
    "-std=c++17",
    "--use_fast_math",
    "-Xcompiler",
    "-fPIC",
    "-Xcompiler",
    "-fvisibility=hidden",
]


# Sources whose elementary functions must be accurate in fp32 (arithmetic of a recurrence, tanh norms, fp32 attention)
ACCURATE = ("attention_any", "delta_rule", "matrix_memory", "tanh_norm")


def _flags(src: Path) -> list[str]:
    return [f for f in NVCC_FLAGS if f != "--use_fast_math" or src.stem not in ACCURATE]


def _nvcc() -> str:
    cand = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(cand):
        raise RuntimeError("nvcc not found; cannot build the sm_100a kernel library")
    return cand


# Sources a model family needs when nothing has been built yet (the whole library otherwise): a fresh checkout
# that only runs this family compiles these into a library of their own.
FAMILY_SOURCES = {
    "latent": ["elementwise", "gemm_simt", "gemm_tcgen05", "latent_attn", "latent_attn_tc", "residual", "sampler"],
    "looped": ["attention", "attention_any", "attention_prefill_tc", "attn_prep", "elementwise", "gemm_simt", "gemm_tcgen05",
               "latent_attn", "latent_attn_tc", "matrix_memory", "moe", "residual", "sampler", "tanh_norm"],
    "prenorm_mix": ["attention", "attention_any", "attention_prefill_tc", "attn_prep", "delta_rule", "elementwise", "gemm_simt",
                    "gemm_tcgen05", "matrix_memory", "moe", "residual", "sampler", "short_conv"],
    "parallel_block": ["attention", "attention_any", "attention_prefill_tc", "attn_prep", "elementwise", "gemm_simt",
                       "gemm_tcgen05", "lightning_attn", "moe", "residual", "sampler"],
}


def _sources(family: str | None = None) -> list[Path]:
    if family is not None:
        return [CSRC / f"{name}.cu" for name in FAMILY_SOURCES[family]]
    return sorted(CSRC.glob("*.cu"))


def _headers() -> list[Path]:
    return sorted(CSRC.glob("*.cuh")) + sorted(CSRC.glob("*.h"))


def _digest(paths: list[Path]) -> str:
    h = hashlib.sha256()
    for p in sorted(paths):
        h.update(p.name.encode())
        h.update(p.read_bytes())
    h.update(" ".join(NVCC_FLAGS).encode() + " ".join(ACCURATE).encode())
    return h.hexdigest()


_active_family: str | None = None      # set when only a family's library is in use (see ensure_kernels)


def lib_path(family: str | None = None) -> Path:
    family = family or _active_family
    return OUT_DIR / (LIB_NAME if family is None else f"libpxl_{family}.so")


def _stamp(family: str | None) -> Path:
    return OUT_DIR / ("build.stamp" if family is None else f"build.{family}.stamp")


def is_fresh(family: str | None = None) -> bool:
    out = OUT_DIR / LIB_NAME if family is None else lib_path(family)
    if not out.exists() or not _stamp(family).exists():
        return False
    return _stamp(family).read_text().strip() == _digest(_sources(family) + _headers())


def ensure_kernels(family: str) -> Path:
    """Kernels for one model family: the whole library if it is built and up to date, else the family's own,
    compiled now if need be. Call before the first kernel of the process runs."""
    global _active_family
    if is_fresh() or family not in FAMILY_SOURCES:
        return build_kernels()
    build_kernels(family=family)
    _active_family = family
    return lib_path()


def build_kernels(force: bool = False, verbose: bool = False, ptxas_info: bool = False,
                  family: str | None = None) -> Path:
    """Compile every ``csrc/*.cu`` (or those of one family) for sm_100a and link them into one shared library."""
    target = OUT_DIR / LIB_NAME if family is None else lib_path(family)
    if not force and is_fresh(family):
        return target
    OUT_DIR.mkdir(parents=True, exist_ok=True)
    obj_dir = OUT_DIR / "obj"
    obj_dir.mkdir(exist_ok=True)
    nvcc = _nvcc()
    srcs = _sources(family)
    if not srcs:
        raise RuntimeError(f"no CUDA sources under {CSRC}")
    headers = _headers()
    hdr_digest = _digest(headers)

    def compile_one(src: Path) -> Path:
        obj = obj_dir / (src.stem + ".o")
        tag = obj_dir / (src.stem + ".tag")
        want = _digest([src]) + hdr_digest
        if not force and obj.exists() and tag.exists() and tag.read_text() == want:
            return obj
        cmd = [nvcc, *_flags(src), "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
        if ptxas_info:
            cmd[1:1] = ["-Xptxas", "-v"]
        res = subprocess.run(cmd, capture_output=True, text=True)
        if verbose or res.returncode != 0:
            sys.stderr.write(res.stdout + res.stderr)
        if res.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src.name}")
        tag.write_text(want)
        return obj

    with ThreadPoolExecutor(max_workers=min(8, len(srcs))) as ex:
        objs = list(ex.map(compile_one, srcs))
    link = [nvcc, "-shared", "-o", str(target), *map(str, objs)]
    res = subprocess.run(link, capture_output=True, text=True)
    if res.returncode != 0:
        sys.stderr.write(res.stdout + res.stderr)
        raise RuntimeError(f"link of {target.name} failed")
    _stamp(family).write_text(_digest(srcs + headers))
    return target


if __name__ == "__main__":
    p = build_kernels(force="--force" in sys.argv, verbose=True, ptxas_info="--ptxas" in sys.argv)
    print(p)
