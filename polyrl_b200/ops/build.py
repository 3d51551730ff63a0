"""In-tree build of the sm_100a extension modules ``polyrl_b200/_serve.so`` and ``polyrl_b200/_C.so``.

Kernel ``.cu`` files are torch-free and compiled directly with ``nvcc -gencode arch=compute_100a,
code=sm_100a -lineinfo``; only the ``bindings*.cpp`` files see torch headers.  The resulting ``.so`` files live in the
package directory (git-ignored; they travel with the tree), never in a JIT cache.

Usage:  python -m polyrl_b200.ops.build [--force] [--verbose]
"""
from __future__ import annotations

import argparse
import concurrent.futures as cf
import os
import subprocess
import sys
import sysconfig
from pathlib import Path

PKG = Path(__file__).resolve().parent.parent
CSRC = PKG / "csrc"
BUILD = CSRC / "build"

# One shared object per module.  ``_serve`` holds what a rollout engine of a mixer stack needs (scheduler, dense GEMMs, packed
# attention, paged decode attention, sampling, sequence mixers); ``_C`` the rest (training, decode GEMMs, multi-GPU).  A kernel
# object may be linked into both.
MODULES: dict[str, dict] = {
    "_serve": {"bindings": "bindings_serve.cpp",
               "cu": ["gemm_tcgen05.cu", "gemm2.cu", "attn_fwd.cu", "decode_attn.cu", "sampling.cu", "mix_elem.cu", "mix_scan.cu", "mix_chunk.cu", "mix_chunk_tc.cu", "mix_delta.cu", "mix_latent.cu",
                      "mix_window.cu", "mix_maps.cu", "mix_block.cu", "mix_experts.cu", "mix_streams.cu", "mix_selective.cu", "mix_gla.cu"]},
    "_C": {"bindings": "bindings.cpp",
           "cu": ["gemm_tcgen05.cu", "gemm2.cu", "skinny_gemm.cu", "decode_gemm.cu", "vmm.cu", "linear_ce.cu", "ag_gemm.cu", "elementwise.cu",
                  "optim.cu", "attn_bwd.cu", "attn_fwd.cu", "p2p.cu", "nvls.cu"]},
}
HEADERS = ["common.cuh", "gemm_sm100.cuh", "gemm2_sm100.cuh", "mixers.cuh", "mix_tc.cuh", "mix_params.hpp"]
HOST_HEADERS = ["kv_manager.hpp", "scheduler.hpp", "bindings_common.hpp", "mix_params.hpp"]          # included by the bindings only
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "--use_fast_math" if False else "-DPRL_NO_FAST_MATH",
    # a function-local static of a kernel launcher (e.g. "attributes are set") belongs to ONE module: launchers linked into both
    # modules must not share it, as GNU unique symbols would across shared objects
    "-Xcompiler", "-fPIC,-fvisibility=hidden,-fno-gnu-unique",
    "--expt-relaxed-constexpr",
]


LAST_BUILD: dict = {}          # what the last build() call did (clean / incremental / up-to-date), printed by __graft_entry__.build()


def _nvcc() -> str:
    cuda_home = os.environ.get("CUDA_HOME", "/usr/local/cuda")
    return str(Path(cuda_home) / "bin" / "nvcc")


def _newer(src: Path, dst: Path, extra: list[Path]) -> bool:
    if not dst.exists():
        return True
    t = dst.stat().st_mtime
    return any(p.stat().st_mtime > t for p in [src, *extra] if p.exists())


def _run(cmd: list[str], verbose: bool) -> None:
    if verbose:
        print(" ".join(cmd), flush=True)
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        sys.stderr.write(r.stdout + r.stderr)
        raise RuntimeError(f"build step failed: {' '.join(cmd[:4])} ...")
    if verbose and (r.stdout or r.stderr):
        print(r.stdout + r.stderr)


def module_path(module: str) -> Path:
    return PKG / f"{module}.so"


def build(force: bool = False, verbose: bool = False, modules: tuple[str, ...] = ("_serve", "_C")) -> Path:
    """Compile what is out of date and link the requested modules; returns the path of the last one."""
    import torch  # noqa: F401  (headers + libs)
    from torch.utils import cpp_extension as ce

    BUILD.mkdir(parents=True, exist_ok=True)
    hdrs = [CSRC / h for h in HEADERS]
    jobs: list[list[str]] = []
    objs: dict[str, list[Path]] = {}
    stale: dict[str, bool] = {}
    queued: set[Path] = set()
    for mod in modules:
        objs[mod], stale[mod] = [], force or not module_path(mod).exists()
        for name in MODULES[mod]["cu"]:
            src = CSRC / name
            obj = BUILD / (src.stem + ".o")
            objs[mod].append(obj)
            if obj in queued:
                stale[mod] = True
            elif force or _newer(src, obj, hdrs):
                jobs.append([_nvcc(), *NVCC_FLAGS, "-I", str(CSRC), "-c", str(src), "-o", str(obj)])
                queued.add(obj)
                stale[mod] = True
        bsrc = CSRC / MODULES[mod]["bindings"]
        bobj = BUILD / (bsrc.stem + ".o")
        objs[mod].append(bobj)
        if force or _newer(bsrc, bobj, [CSRC / h for h in HOST_HEADERS]):
            inc = []
            for p in ce.include_paths("cuda") if "device_type" in ce.include_paths.__code__.co_varnames else ce.include_paths(True):
                inc += ["-isystem", p]
            inc += ["-isystem", sysconfig.get_paths()["include"]]
            jobs.insert(0, [
                "g++", "-O2", "-std=c++17", "-fPIC", "-fvisibility=hidden", "-fno-gnu-unique", f"-DTORCH_EXTENSION_NAME={mod}", "-DTORCH_API_INCLUDE_EXTENSION_H",
                f"-D_GLIBCXX_USE_CXX11_ABI={int(torch._C._GLIBCXX_USE_CXX11_ABI)}", *inc, "-c", str(bsrc), "-o", str(bobj),
            ])
            stale[mod] = True
        so = module_path(mod)
        stale[mod] = stale[mod] or any(o.exists() and so.exists() and o.stat().st_mtime > so.stat().st_mtime for o in objs[mod])
    import time

    t0 = time.time()
    if jobs:
        with cf.ThreadPoolExecutor(max_workers=min(max(2, os.cpu_count() or 2), 16, len(jobs))) as ex:
            list(ex.map(lambda c: _run(c, verbose), jobs))
    global LAST_BUILD
    total = len({o for v in objs.values() for o in v})
    LAST_BUILD = {"build_mode": "clean" if len(jobs) == total else ("incremental" if jobs else "up-to-date"), "modules": list(modules),
                  "objects_compiled": len(jobs), "objects_total": total, "compile_s": round(time.time() - t0, 1),
                  "arch": "compute_100a/sm_100a", "nvcc_flags": NVCC_FLAGS}
    for mod in modules:
        if not stale[mod]:
            continue
        out = module_path(mod)
        lib_dirs = ce.library_paths("cuda") if "device_type" in ce.library_paths.__code__.co_varnames else ce.library_paths(True)
        tmp_out = out.with_suffix(f".so.tmp{os.getpid()}")     # link next to the target, then rename: readers never see a half-written .so
        link = ["g++", "-shared", "-o", str(tmp_out), *map(str, objs[mod])]
        for d in lib_dirs:
            link += [f"-L{d}", f"-Wl,-rpath,{d}"]
        link += ["-lc10", "-lc10_cuda", "-ltorch_cpu", "-ltorch_cuda", "-ltorch", "-ltorch_python", "-lcudart"]
        _run(link, verbose)
        tmp_out.replace(out)
    return module_path(modules[-1])


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--verbose", action="store_true")
    ap.add_argument("--modules", default="_serve,_C", help="comma-separated subset of the modules to build")
    a = ap.parse_args()
    print(build(a.force, a.verbose, tuple(a.modules.split(","))))
    import json

    print(json.dumps(LAST_BUILD))


if __name__ == "__main__":
    main()
