"""Native libraries and how they are compiled (nvcc, sm_100a, in-tree).

``build(name)`` compiles one library if it is missing or older than its sources; every source is
its own nvcc process, so a library takes as long as its slowest file.  The llama megakernel and
the hybrid models' kernels are separate libraries: a user of one does not compile the other.
Run as ``python -m megakernels_b200.build [name ...]``.
"""

from __future__ import annotations

import os
import subprocess
import sys
import tempfile
from concurrent.futures import ThreadPoolExecutor
from dataclasses import dataclass
from pathlib import Path

PACKAGE = Path(__file__).resolve().parent
CSRC = PACKAGE / "csrc"
NATIVE = PACKAGE / "native"
INCLUDE = PACKAGE.parent / "include"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC",
]


@dataclass(frozen=True)
class Library:
    output: str
    sources: tuple[str, ...]
    headers: tuple[str, ...]  # relative to csrc

    @property
    def path(self) -> Path:
        return NATIVE / self.output

    def stale(self) -> bool:
        if not self.path.exists():
            return True
        built = self.path.stat().st_mtime
        return any((CSRC / n).stat().st_mtime > built for n in self.sources + self.headers)


LIBRARIES = {
    "llama": Library(
        "libmkb200.so",
        ("megakernel.cu", "megakernel_batched.cu", "megakernel_gemm.cu", "host.cu", "no_alloc.cu", "peer.cu"),
        ("mk_common.cuh", "megakernel.cu", "../../include/mkb200.h"),
    ),
    "hybrid": Library(
        "libmkb200_hybrid.so",
        ("hybrid_decode.cu", "hybrid_decode_rotary.cu", "hybrid_decode_mixed.cu", "hybrid_prefill.cu",
         "hybrid_attention.cu", "hybrid_flash.cu", "hybrid_gemm_bf16.cu", "hybrid_gemm_f32.cu", "hybrid_host.cu"),
        ("hybrid_common.cuh", "hybrid_kernels.h", "hybrid_decode.cu", "hybrid_tcgen05.cuh", "mk_common.cuh", "../../include/mkb200.h",
         "../../include/mkb200_hybrid.h"),
    ),
}


def build(name: str, quiet: bool = False) -> Path:
    """Compile library ``name`` if it is stale; returns its path."""
    lib = LIBRARIES[name]
    if not lib.stale():
        return lib.path
    nvcc = os.environ.get("NVCC", "nvcc")
    with tempfile.TemporaryDirectory(dir=NATIVE, prefix=".build-") as tmp:
        def compile_one(src: str) -> str:
            obj = str(Path(tmp) / (Path(src).stem + ".o"))
            cmd = [nvcc, *NVCC_FLAGS, "-c", "-o", obj, str(CSRC / src)]
            if not quiet:
                print(" ".join(cmd), file=sys.stderr, flush=True)
            run = subprocess.run(cmd, cwd=str(CSRC), stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
            if run.returncode:
                raise RuntimeError(f"{' '.join(cmd)} failed:\n{run.stdout}")
            return obj

        with ThreadPoolExecutor(max_workers=len(lib.sources)) as pool:
            objects = list(pool.map(compile_one, lib.sources))
        part = str(Path(tmp) / lib.output)
        run = subprocess.run([nvcc, *NVCC_FLAGS[:2], "-shared", "-o", part, *objects],
                             stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
        if run.returncode:
            raise RuntimeError(f"linking {lib.output} failed:\n{run.stdout}")
        os.replace(part, lib.path)
    return lib.path


if __name__ == "__main__":
    for target in sys.argv[1:] or LIBRARIES:
        print(build(target))
