"""Build the C-ABI CUDA library in-tree with nvcc for sm_100a.

``python -m spikeinfer_b200.build`` compiles ``csrc/*.cu`` into
``spikeinfer_b200/libspikeinfer_b200.so``.  nvcc cross-compiles without a GPU, so this
also runs on a CPU-only build machine.  The library is rebuilt only when a source or
header is newer than it (``force=True`` overrides).  :func:`build_components` builds a library of some of
the translation units only, for a process that serves one kind of model from a fresh checkout.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys
from pathlib import Path

PKG_DIR = Path(__file__).resolve().parent
CSRC = PKG_DIR / "csrc"
INCLUDE = PKG_DIR.parent / "include"
LIB_PATH = PKG_DIR / "libspikeinfer_b200.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-O3", "-std=c++17", "-lineinfo",
    "-Xcompiler", "-fPIC",
]
# Translation units whose arithmetic contract forbids contracting a multiply and an add into one rounding: the LIF
# recurrence (every product and sum is rounded on its own, as the reference does) and the RMSNorm's mean + eps.
NO_FMA_CONTRACTION = {"spk_lif.cu", "spk_norm.cu"}

# Groups of translation units a model may need; "core" (C ABI basics, batch metadata, sampling) is part of every library.
COMPONENTS = {
    "core": ("spk_capi.cu", "spk_meta.cu", "spk_sample.cu"),
    "spike": ("spk_attn.cu", "spk_attn_stream.cu", "spk_lif.cu", "spk_norm.cu", "spk_pack.cu"),
    "dense": ("spk_postnorm.cu", "spk_paged_attn.cu", "spk_sigmoid_prefill.cu", "spk_sigmoid_decode.cu", "spk_decay.cu",
              "spk_decay_mma.cu"),
    "latent": ("spk_prenorm.cu", "spk_experts.cu", "spk_experts_mma.cu", "spk_latent.cu", "spk_latent_decode.cu",
               "spk_latent_prefill.cu", "spk_delta.cu", "spk_delta_mma.cu"),
}


def _nvcc() -> str:
    exe = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(exe):
        raise RuntimeError("nvcc not found: the CUDA library cannot be built")
    return exe


def sources(components=None) -> list[Path]:
    if components is None:
        return sorted(CSRC.glob("*.cu"))
    names = {n for c in {"core", *components} for n in COMPONENTS[c]}
    return sorted(CSRC / n for n in names)


def library_path(components=None) -> Path:
    if components is None:
        return LIB_PATH
    return PKG_DIR / f"libspikeinfer_b200.{'-'.join(sorted({'core', *components}))}.so"


def is_stale(components=None) -> bool:
    lib = library_path(components)
    if not lib.exists():
        return True
    built = lib.stat().st_mtime
    deps = sources(components) + list(CSRC.glob("*.cuh")) + list(INCLUDE.glob("*.h"))
    return any(p.stat().st_mtime > built for p in deps)


def build_components(components) -> Path:
    """The library to load for these components: the full one when it is there and current, else one of their
    translation units alone, compiled on first use."""
    if not is_stale():
        return LIB_PATH
    return build(components=tuple(components))


def build(force: bool = False, verbose: bool = False, ptxas_info: bool = False, components=None) -> Path:
    lib_path = library_path(components)
    if not force and not is_stale(components):
        return lib_path
    obj_dir = PKG_DIR / "build"
    obj_dir.mkdir(exist_ok=True)
    nvcc = _nvcc()
    objs = []
    procs = []
    for src in sources(components):
        obj = obj_dir / (src.stem + ".o")
        cmd = [nvcc, *NVCC_FLAGS, "-I", str(INCLUDE), "-c", str(src), "-o", str(obj)]
        if src.name in NO_FMA_CONTRACTION:
            cmd.insert(1, "--fmad=false")
        if ptxas_info:
            cmd[1:1] = ["-Xptxas", "-v"]
        if verbose:
            print(" ".join(cmd), flush=True)
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
        objs.append(obj)
    failed = []
    for src, proc in procs:
        out, _ = proc.communicate()
        if proc.returncode != 0:
            failed.append(f"--- {src.name} ---\n{out}")
        elif (verbose or ptxas_info) and out.strip():
            print(f"--- {src.name} ---\n{out}", flush=True)
    if failed:
        raise RuntimeError("nvcc failed:\n" + "\n".join(failed))
    tmp = lib_path.with_suffix(".so.tmp")
    link = [nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-o", str(tmp),
            *map(str, objs), "-lcudart", "-ldl"]
    if verbose:
        print(" ".join(link), flush=True)
    subprocess.run(link, check=True)
    os.replace(tmp, lib_path)
    return lib_path


if __name__ == "__main__":
    path = build(force="--force" in sys.argv, verbose="-v" in sys.argv, ptxas_info="--ptxas" in sys.argv)
    print(path)
