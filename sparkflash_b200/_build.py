"""In-tree native build.

Four shared libraries with a plain C ABI (loaded through ctypes, see ``_lib.py``), each built on its own when it is first
needed, so that a model compiles what it uses:

* ``lib/libsfb_core.so``  - g++: what every model needs - scheduler core, radix cache and page allocator, safetensors and
  rank-file reader.
* ``lib/libsfb_host.so``  - g++: codecs, CPU oracle ops, speculation policy, constrained-decoding automaton, Engram hash.
* ``lib/libsfb_rows.so``  - nvcc for sm_100a only: kernels of the layered decoders (models/layered.py) and the sampler.
* ``lib/libsfb_cuda.so``  - nvcc for sm_100a only: every other device kernel and its launcher, the
  symmetric-memory helpers and the lane (virtual memory) allocator.

Objects are rebuilt only when the hash of the source (plus headers and flags) changes, so importing
the package on a machine that received the built tree does not compile anything.
"""
from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

ROOT = Path(__file__).resolve().parent
CSRC = ROOT / "csrc"
LIBDIR = ROOT / "lib"
OBJDIR = ROOT / "lib" / "obj"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC", "-Xptxas", "-v", "--expt-relaxed-constexpr",
    "-Xcompiler", "-Wno-unused-function",
]
if os.environ.get("SFB_KERNEL_MARKS") == "1":      # in-kernel phase marks (utils/kernel_marks.py): a measurement build
    NVCC_FLAGS.append("-DSFB_KERNEL_MARKS")
_CORE = ("host_sched.cpp", "host_radix.cpp", "host_weights.cpp")


def _sources(lib: str) -> list[Path]:
    cu, cpp = sorted(CSRC.rglob("*.cu")), sorted(CSRC.rglob("*.cpp"))
    return {"core": [s for s in cpp if s.name in _CORE],
            "host": [s for s in cpp if s.name not in _CORE],
            "rows": [s for s in cu if s.name.startswith("k_rows") or s.name == "k_sample.cu"],
            "cuda": [s for s in cu if not s.name.startswith("k_rows")]}[lib]


LIBRARIES = ("core", "host", "rows", "cuda")
GXX_FLAGS = ["-O2", "-std=c++17", "-fPIC", "-Wall", "-Wno-unused-function", "-pthread"]


def _nvcc() -> str:
    for cand in (os.environ.get("SFB_NVCC"), "/usr/local/cuda/bin/nvcc", shutil.which("nvcc")):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found (set SFB_NVCC)")


def _headers_digest() -> str:
    h = hashlib.sha256()
    for p in sorted(list(CSRC.rglob("*.h")) + list(CSRC.rglob("*.cuh"))):
        h.update(p.name.encode())
        h.update(p.read_bytes())
    return h.hexdigest()


def _digest(src: Path, flags: list[str], hdr: str) -> str:
    h = hashlib.sha256()
    h.update(src.read_bytes())
    h.update(" ".join(flags).encode())
    h.update(hdr.encode())
    return h.hexdigest()


def _compile_one(cmd: list[str], src: Path, obj: Path, stamp: Path, digest: str, verbose: bool) -> str:
    if obj.exists() and stamp.exists() and stamp.read_text() == digest:
        return f"[up-to-date] {src.name}"
    r = subprocess.run(cmd, capture_output=True, text=True)
    log = OBJDIR / (src.name + ".log")
    log.write_text(r.stdout + r.stderr)
    if r.returncode != 0:
        raise RuntimeError(f"compile failed: {' '.join(cmd)}\n{r.stdout}\n{r.stderr}")
    stamp.write_text(digest)
    if verbose:
        sys.stderr.write(r.stderr)
    return f"[built] {src.name}"


def build(verbose: bool = False, force: bool = False, only: tuple[str, ...] | None = None) -> dict[str, Path]:
    """Compile the native sources for sm_100a / the host and link the libraries (``only``: names out of LIBRARIES)."""
    names = tuple(only or LIBRARIES)
    LIBDIR.mkdir(exist_ok=True)
    OBJDIR.mkdir(exist_ok=True)
    hdr = _headers_digest()
    jobs, objs = {}, {n: [] for n in names}
    for n in names:
        for s in _sources(n):
            cuda = s.suffix == ".cu"
            cc, flags = (_nvcc(), NVCC_FLAGS) if cuda else ("g++", GXX_FLAGS)
            o = OBJDIR / (s.name + ".o")
            objs[n].append(o)
            jobs[s.name] = ([cc, *flags, "-I", str(CSRC), "-c", str(s), "-o", str(o)], s, o, OBJDIR / (s.name + ".stamp"), _digest(s, flags, hdr))
    if force:
        for j in jobs.values():
            if j[3].exists():
                j[3].unlink()
    with ThreadPoolExecutor(max_workers=max(2, (os.cpu_count() or 4))) as ex:
        results = dict(zip(jobs, ex.map(lambda j: _compile_one(*j, verbose), jobs.values())))
    if verbose:
        print("\n".join(results.values()))
    out = {}
    for n in names:
        so = LIBDIR / f"libsfb_{n}.so"
        out[n] = so
        stamp = OBJDIR / f"lib{n}.stamp"
        want = hashlib.sha256(" ".join(j[4] for j in (jobs[s.name] for s in _sources(n))).encode()).hexdigest()
        if so.exists() and stamp.exists() and stamp.read_text() == want:
            continue
        part = LIBDIR / f".libsfb_{n}.{os.getpid()}.so"      # linked beside, then renamed: a reader never sees half a file
        if n in ("core", "host"):
            cmd = ["g++", "-shared", "-o", str(part), *map(str, objs[n]), "-pthread"]
        else:
            cmd = [_nvcc(), "-shared", "-o", str(part), *map(str, objs[n]), "-gencode", "arch=compute_100a,code=sm_100a", "-Xcompiler", "-fPIC"]
        subprocess.run(cmd, check=True, capture_output=True)
        os.replace(part, so)
        stamp.write_text(want)
    return out


def ptxas_report() -> str:
    """Registers / spills / shared memory per kernel, as printed by ``-Xptxas -v`` at build."""
    out = []
    for log in sorted(OBJDIR.glob("*.cu.log")):
        out.append(f"== {log.name}")
        out.append(log.read_text())
    return "\n".join(out)


if __name__ == "__main__":
    libs = build(verbose="-v" in sys.argv, force="-f" in sys.argv)
    for k, v in libs.items():
        print(k, v, v.stat().st_size)
