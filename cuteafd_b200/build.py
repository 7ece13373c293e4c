"""Builds the native library in-tree: every `csrc/*.cu` is compiled for sm_100a with nvcc and linked into
`cuteafd_b200/_native/libcuteafd_b200.so`.  No GPU is needed (nvcc cross-compiles); objects are rebuilt
only when their source or a header is newer.  `python -m cuteafd_b200.build [--force] [--verbose]`.

The reference builds its native library with CMake (native/CMakeLists.txt); here one small Python driver is
enough because there are no AOT-exported objects to stitch in.
"""
from __future__ import annotations

import argparse
import hashlib
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

ROOT = Path(__file__).resolve().parent
CSRC = ROOT / "csrc"
OUT = ROOT / "_native"
LIB = OUT / "libcuteafd_b200.so"
STAMP = OUT / "build" / "full.stamp"        # hash of the sources the full library was built from

# what one family's single-GPU engine launches: enough for a checkout that only serves that family
SUBSETS = {"latent_stack": (["runtime", "elementwise", "moe", "sampling", "tc_gemm", "attention_mla", "attention_mla_prefill", "latent_stack", "f32_linear"],
                            ["-DCA_TC_BF16_ONLY"]),
           "hybrid_stack": (["runtime", "elementwise", "sampling", "tc_gemm", "attention_tc", "attention_mla_prefill", "hybrid_stack", "f32_linear"],
                            ["-DCA_TC_BF16_ONLY"]),
           "hyper_stack": (["runtime", "elementwise", "moe", "sampling", "tc_gemm", "attention_tc", "attention_mla_prefill", "hybrid_stack", "hyper_stack", "decay_scan", "f32_linear"],
                           ["-DCA_TC_BF16_ONLY"]),
           "mixed_stack": (["runtime", "elementwise", "sampling", "tc_gemm", "attention_tc", "attention_mla", "attention_mla_prefill", "hybrid_stack", "latent_stack", "hyper_stack", "decay_scan",
                            "mixed_stack", "f32_linear"], ["-DCA_TC_BF16_ONLY"])}

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "--use_fast_math=false", "-Xptxas", "-v"]


def nvcc_path() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found")


def _stale(obj: Path, src: Path, headers: list[Path]) -> bool:
    if not obj.exists():
        return True
    t = obj.stat().st_mtime
    return any(p.stat().st_mtime > t for p in [src, *headers])


def source_hash(stems: list[str] | None = None, extra: list[str] | None = None) -> str:
    """Of the sources (all, or the named ones), every header and the compiler flags: says whether a built library is current wherever the
    tree was copied to (time stamps do not survive every copy)."""
    h = hashlib.sha256(repr((NVCC_FLAGS, extra or [])).encode())
    files = sorted(CSRC.glob("*.cuh")) + sorted(CSRC.glob("*.h")) + [p for p in sorted(CSRC.glob("*.cu")) if stems is None or p.stem in stems]
    for p in files:
        h.update(p.name.encode() + p.read_bytes())
    return h.hexdigest()[:16]


def ensure(subset: str | None = None) -> Path:
    """A current library: the full one when it was built from these sources, else the named subset (built on first use), else a full build."""
    if LIB.exists() and STAMP.exists() and STAMP.read_text() == source_hash():
        return LIB
    if subset is None:
        return build()
    stems, extra = SUBSETS[subset]
    out = OUT / f"libcuteafd_b200_{subset}_{source_hash(stems, extra)}.so"
    if not out.exists():
        work = OUT / "build" / f"{subset}-{os.getpid()}"
        work.mkdir(parents=True, exist_ok=True)
        flags = [f for f in NVCC_FLAGS if f != "--use_fast_math=false"] + extra

        def compile_one(stem):
            return stem, subprocess.run([nvcc_path(), *flags, "-I", str(CSRC), "-c", str(CSRC / f"{stem}.cu"), "-o", str(work / f"{stem}.o")],
                                        capture_output=True, text=True)
        with ThreadPoolExecutor(max_workers=min(len(stems), os.cpu_count() or 4)) as ex:
            for stem, r in ex.map(compile_one, stems):
                if r.returncode != 0:
                    sys.stderr.write(f"--- {stem}.cu\n{r.stdout}{r.stderr}\n")
                    raise RuntimeError(f"nvcc failed on {stem}.cu")
        tmp = work / out.name
        r = subprocess.run([nvcc_path(), "-shared", "--cudart", "shared", "-o", str(tmp), *[str(work / f"{s}.o") for s in stems]], capture_output=True, text=True)
        if r.returncode != 0:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError("link failed")
        os.replace(tmp, out)
        shutil.rmtree(work, ignore_errors=True)
    return out


def build(force: bool = False, verbose: bool = False) -> Path:
    OUT.mkdir(exist_ok=True)
    nvcc = nvcc_path()
    headers = sorted(CSRC.glob("*.cuh")) + sorted(CSRC.glob("*.h"))
    sources = sorted(CSRC.glob("*.cu"))
    flags = [f for f in NVCC_FLAGS if f != "--use_fast_math=false"]
    jobs = []
    for src in sources:
        obj = OUT / (src.stem + ".o")
        if force or _stale(obj, src, headers):
            jobs.append((src, obj))

    def compile_one(job):
        src, obj = job
        cmd = [nvcc, *flags, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        return src, r

    if jobs:
        with ThreadPoolExecutor(max_workers=min(len(jobs), os.cpu_count() or 4)) as ex:
            for src, r in ex.map(compile_one, jobs):
                if verbose or r.returncode != 0:
                    sys.stderr.write(f"--- {src.name}\n{r.stdout}{r.stderr}\n")
                if r.returncode != 0:
                    raise RuntimeError(f"nvcc failed on {src.name}")
    objs = [OUT / (s.stem + ".o") for s in sources]
    if force or jobs or not LIB.exists():
        cmd = [nvcc, "-shared", "--cudart", "shared", "-o", str(LIB), *map(str, objs)]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError("link failed")
    if force or jobs or not STAMP.exists():
        STAMP.parent.mkdir(exist_ok=True)
        STAMP.write_text(source_hash())
    return LIB


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--force", action="store_true")
    ap.add_argument("--verbose", action="store_true")
    a = ap.parse_args()
    print(build(a.force, a.verbose))


if __name__ == "__main__":
    main()
