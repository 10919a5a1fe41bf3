"""Builds liblbk.so (the CUDA C-ABI library) in-tree with nvcc for sm_100a."""
from __future__ import annotations

import os
import shutil
import subprocess
from pathlib import Path

PKG = Path(__file__).resolve().parent
ROOT = PKG.parent
CSRC = PKG / "csrc"
LIB = PKG / "liblbk.so"
OBJ = PKG / "_build"  # object files (git-ignored)

# The runtime every model family needs, and what each family adds. liblbk.so holds all of it; a process that only
# serves one family can do with that family's part (library_for).
RUNTIME = ["lbk_context.cu", "lbk_bf16.cu", "lbk_decoder.cu", "lbk_attn_tc.cu", "lbk_model.cu"]
FAMILIES = {
    "": ["lbk_api.cu", "lbk_gemv.cu", "lbk_quant.cu", "lbk_plan.cu", "lbk_sweep.cu", "lbk_gemm.cu", "lbk_noalloc.cu", "lbk_tp.cu",
         "lbk_bitnet.cu", "lbk_convert.cu", "lbk_probe.cu"],
    "Pefolix": ["lbk_layernorm.cu", "lbk_dense.cu", "lbk_moe.cu", "lbk_attn_window.cu", "lbk_pefolix.cu"],
    "Dugulorn": ["lbk_layernorm.cu", "lbk_dense.cu", "lbk_attn_window.cu", "lbk_latent.cu", "lbk_recur.cu", "lbk_dugulorn.cu"],
}
SOURCES = RUNTIME + list(dict.fromkeys(s for f in FAMILIES.values() for s in f))  # families share kernel files
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
]


def nvcc_path() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found; liblbk.so cannot be built")


def is_stale(lib: Path = None) -> bool:
    lib = lib or LIB
    if not lib.exists():
        return True
    t = lib.stat().st_mtime
    deps = list(CSRC.glob("*.cu")) + list(CSRC.glob("*.cuh")) + [ROOT / "include" / "lbk.h"]
    return any(d.stat().st_mtime > t for d in deps)


def _run(cmd, env):
    res = subprocess.run(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True, env=env)
    if res.returncode != 0:
        raise RuntimeError("nvcc failed:\n" + " ".join(cmd) + "\n" + res.stdout)
    return res.stdout


def library_for(architecture: str) -> Path:
    """The library a process that serves this one family loads: liblbk.so when it is built and fresh, else
    liblbk-<architecture>.so, compiled now from the runtime and the family's own sources."""
    if not is_stale():
        return LIB
    if architecture not in FAMILIES or architecture == "":
        return build()
    return build(lib=PKG / f"liblbk-{architecture}.so", sources=RUNTIME + FAMILIES[architecture])


def build(force: bool = False, verbose: bool = False, lib: Path = None, sources=None) -> Path:
    """Compile every .cu (one object each, side by side, only the ones whose source or any header
    changed) and link lemonade_burn_b200/liblbk.so (or `lib` from `sources`). Returns the library path."""
    lib, sources = lib or LIB, sources or SOURCES
    if not force and not is_stale(lib):
        return lib
    from concurrent.futures import ThreadPoolExecutor
    OBJ.mkdir(exist_ok=True)
    env = dict(os.environ)
    env.pop("CC", None)
    env.pop("CXX", None)
    nvcc = nvcc_path()
    headers = list(CSRC.glob("*.cuh")) + [ROOT / "include" / "lbk.h"]
    newest_header = max(h.stat().st_mtime for h in headers)
    jobs = []
    for s in sources:
        src, obj = CSRC / s, OBJ / (Path(s).stem + ".o")
        if force or not obj.exists() or obj.stat().st_mtime < max(src.stat().st_mtime, newest_header):
            cmd = [nvcc, *NVCC_FLAGS, "-c", f"-I{ROOT / 'include'}", f"-I{CSRC}", "-o", str(obj), str(src)]
            if verbose:
                cmd += ["-Xptxas", "-v"]
            jobs.append(cmd)
    with ThreadPoolExecutor(max_workers=min(len(jobs), os.cpu_count() or 4) or 1) as pool:
        logs = list(pool.map(lambda c: _run(c, env), jobs))
    if verbose:
        print("\n".join(logs))
    part = lib.with_name(f".{lib.name}.{os.getpid()}")  # a half-written library is never loaded
    _run([nvcc, "-shared", "-o", str(part)] + [str(OBJ / (Path(s).stem + ".o")) for s in sources], env)
    os.replace(part, lib)
    return lib


if __name__ == "__main__":
    import sys

    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
