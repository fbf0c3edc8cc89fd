"""In-tree build of the native libraries: one nvcc call each, sm_100a only.

    python -m tilert_b200.build

writes ``tilert_b200/libtilert_b200.so`` and ``tilert_b200/libtilert_gqa.so`` next to the package (the place
``load_backend`` looks), and the dispatcher registration library.
"""

from __future__ import annotations

import os
import re
import shutil
import subprocess
import sys
import tempfile
from dataclasses import dataclass
from pathlib import Path

PKG = Path(__file__).resolve().parent
NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-shared", "-Xcompiler", "-fPIC",
]


@dataclass(frozen=True)
class Target:
    src: Path
    out: Path
    flags: tuple[str, ...] = ()


# The libraries share headers with kernels in them: the second one binds its own definitions (-Bsymbolic), whatever
# else is loaded in the process.
TARGETS = {
    "deepseek_v3_2": Target(PKG / "csrc" / "cabi.cu", PKG / "libtilert_b200.so"),
    "ralasun": Target(PKG / "csrc" / "gqa_cabi.cu", PKG / "libtilert_gqa.so", ("-Xlinker", "-Bsymbolic")),
}
SRC, OUT = TARGETS["deepseek_v3_2"].src, TARGETS["deepseek_v3_2"].out

BIND_SRC = PKG / "csrc" / "torch_binding.cpp"
BIND_OUT = PKG / "libtilert_dsv32.so"


def build_binding(force: bool = False) -> Path:
    """The dispatcher registration library (TORCH_LIBRARY translation unit over the C ABI): g++ against the
    installed torch headers, linked to libtilert_b200.so next to it."""
    import torch

    if not force and BIND_OUT.exists() and BIND_OUT.stat().st_mtime >= max(BIND_SRC.stat().st_mtime, OUT.stat().st_mtime):
        return BIND_OUT
    t = Path(torch.__file__).resolve().parent
    cuda_inc = "/usr/local/cuda/include"
    cmd = ["g++", "-O2", "-std=c++17", "-shared", "-fPIC", f"-D_GLIBCXX_USE_CXX11_ABI={int(torch._C._GLIBCXX_USE_CXX11_ABI)}",
           f"-I{t / 'include'}", f"-I{t / 'include' / 'torch' / 'csrc' / 'api' / 'include'}", f"-I{cuda_inc}", str(BIND_SRC),
           "-o", str(BIND_OUT), f"-L{t / 'lib'}", "-ltorch", "-ltorch_cpu", "-lc10", "-lc10_cuda", f"-L{PKG}",
           "-l:libtilert_b200.so", "-Wl,-rpath,$ORIGIN"]
    res = subprocess.run(cmd, capture_output=True, text=True)
    if res.returncode != 0:
        raise RuntimeError(f"g++ failed:\n{res.stdout}\n{res.stderr}")
    return BIND_OUT


def sources(src: Path, seen: set[Path] | None = None) -> set[Path]:
    """``src`` and every in-tree file it includes."""
    seen = set() if seen is None else seen
    src = src.resolve()
    if src not in seen and src.exists():
        seen.add(src)
        for name in re.findall(r'^#include "([^"]+)"', src.read_text(), flags=re.M):
            sources(src.parent / name, seen)
    return seen


def needs_build(model_type: str = "deepseek_v3_2") -> bool:
    t = TARGETS[model_type]
    return not t.out.exists() or max(p.stat().st_mtime for p in sources(t.src)) > t.out.stat().st_mtime


def nvcc() -> str:
    return shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"


def build(force: bool = False, verbose: bool = False, model_type: str = "deepseek_v3_2") -> Path:
    t = TARGETS[model_type]
    if not force and not needs_build(model_type):
        return t.out
    fd, part = tempfile.mkstemp(dir=t.out.parent, prefix=f".{t.out.name}.")
    os.close(fd)
    try:
        cmd = [nvcc(), *NVCC_FLAGS, *t.flags, *(["-Xptxas", "-v"] if verbose else []), "-o", part, str(t.src)]
        res = subprocess.run(cmd, capture_output=True, text=True)
        if res.returncode != 0:
            raise RuntimeError(f"nvcc failed:\n{res.stdout}\n{res.stderr}")
        os.chmod(part, 0o755)
        os.replace(part, t.out)  # a process that is loading the old file keeps it
    finally:
        if os.path.exists(part):
            os.unlink(part)
    if verbose:
        print(res.stderr)
    return t.out


if __name__ == "__main__":
    for name in TARGETS:
        print(build(force=True, verbose="-v" in sys.argv, model_type=name))
    print(build_binding(force=True))
