"""Builds the C-ABI library ``libb200llm.so`` in-tree with nvcc for sm_100a.

Each ``csrc/*.cu`` is compiled to an object next to the library and relinked only when its source
(or a shared header) is newer, so a rebuild after touching one kernel takes seconds.  nvcc
cross-compiles without a GPU.  Run ``python -m llm_from_scratch_b200._build`` or call ``build()``.
"""
from __future__ import annotations

import fcntl
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
INCLUDE = PKG.parent / "include"
OBJ_DIR = PKG / "build"
LIB_PATH = PKG / "libb200llm.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo",
    "-Xcompiler", "-fPIC",
    "--expt-relaxed-constexpr",
    "-Xptxas", "-v",
]


def _nvcc() -> str:
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found: the CUDA kernels cannot be built")
    return exe


def _stale(target: Path, deps: list[Path]) -> bool:
    if not target.exists():
        return True
    t = target.stat().st_mtime
    return any(d.stat().st_mtime > t for d in deps)


# Sources a model family runs on, where that is not the whole library: ``ensure`` builds a library of just these
# when the full one is absent.  "api" and "host_path" are the parts every engine uses.
FAMILY_SOURCES = {
    "Nabalix": ("api", "host_path", "decode_advance", "sampler", "moe_gemm", "moe_gemm_rows", "grouped_linear", "store_kvcache", "prefill_plan", "streams",
                "talking_attention", "talking_attention_mma", "talking_decode_mma", "gated_recurrence"),
    "Taminex": ("api", "host_path", "decode_advance", "sampler", "moe_gemm", "moe_gemm_rows", "grouped_linear", "store_kvcache", "prefill_plan",
                "prefill_varlen", "prefill_mma", "prefill_umma", "prefill_umma2", "prefill_umma4", "paged_decode", "mla_decode",
                "mla_decode_mma", "residual_norm", "head_norm_rope", "latent_rows", "activations", "delta_rule", "delta_chunk"),
    "Meresun": ("api", "host_path", "decode_advance", "sampler", "moe_gemm", "moe_gemm_rows", "grouped_linear", "moe_group_route",
                "store_kvcache", "prefill_plan", "prefill_varlen", "prefill_mma", "prefill_umma", "prefill_umma2", "prefill_umma4",
                "paged_decode", "mla_decode", "mla_decode_mma", "residual_norm", "gated_residual", "latent_rows", "activations"),
    "Sodonex": ("api", "host_path", "decode_advance", "sampler", "moe_gemm", "moe_gemm_rows", "grouped_linear", "moe_group_route",
                "store_kvcache", "prefill_plan", "prefill_varlen", "prefill_mma", "prefill_umma", "prefill_umma2", "prefill_umma4",
                "paged_decode", "latent_rows", "activations", "shift_residual", "conv_norm_rope"),
}


def _headers() -> list[Path]:
    return sorted(CSRC.glob("*.cuh")) + sorted(INCLUDE.glob("*.h")) + [Path(__file__)]


def ensure(family: str | None = None) -> Path:
    """A library that can run ``family`` (an ``architecture`` name), built if need be: the full library when it
    is there and current, else one of the family's sources only.  Sets ``B200LLM_LIBRARY`` for ``_lib``."""
    sources = sorted(CSRC.glob("*.cu"))
    if not _stale(LIB_PATH, sources + _headers()) or family not in FAMILY_SOURCES:
        path = build()
    else:
        names = FAMILY_SOURCES[family]
        path = build(sources=[CSRC / f"{n}.cu" for n in names], target=PKG / f"libb200llm_{family.lower()}.so")
    os.environ["B200LLM_LIBRARY"] = str(path)
    return path


def build(force: bool = False, verbose: bool = False, sources: list[Path] | None = None,
          target: Path | None = None) -> Path:
    """Compile every kernel source and link ``libb200llm.so`` (or the given sources into ``target``); returns its
    path.  Builds of one checkout take turns."""
    OBJ_DIR.mkdir(exist_ok=True)
    with open(OBJ_DIR / "lock", "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        return _build_locked(force, verbose, sources or sorted(CSRC.glob("*.cu")), target or LIB_PATH)


def _build_locked(force: bool, verbose: bool, sources: list[Path], target: Path) -> Path:
    nvcc = _nvcc()
    headers = _headers()
    jobs = []
    for src in sources:
        obj = OBJ_DIR / (src.stem + ".o")
        if force or _stale(obj, [src] + headers):
            jobs.append((src, obj))

    def compile_one(job):
        src, obj = job
        cmd = [nvcc, *NVCC_FLAGS, "-I", str(INCLUDE), "-c", str(src), "-o", str(obj)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        log = OBJ_DIR / (src.stem + ".ptxas.log")
        log.write_text(r.stderr)
        if r.returncode != 0:
            raise RuntimeError(f"nvcc failed for {src.name}:\n{r.stdout}\n{r.stderr}")
        if verbose:
            sys.stderr.write(r.stderr)
        return obj

    if jobs:
        with ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            list(ex.map(compile_one, jobs))
    objs = [OBJ_DIR / (s.stem + ".o") for s in sources]
    if force or jobs or _stale(target, objs):
        cmd = [nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a",
               "-o", str(target), *map(str, objs)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    return target


if __name__ == "__main__":
    path = build(force="--force" in sys.argv, verbose="-v" in sys.argv)
    print(path)
