"""Build libzipage_b200.so (sm_100a) in-tree with nvcc.

`python -m zipage_b200.build` compiles every csrc/*.cu to an object file (in
parallel) and links them into zipage_b200/libzipage_b200.so next to this file.
No GPU is needed to build.  Objects are rebuilt only when a source or header
is newer than the object.

A model family needs only some of the sources: `ensure(part)` hands out the full library when it is
current and otherwise builds (once) a smaller one from that family's sources.
"""
from __future__ import annotations

import fcntl
import hashlib
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG = Path(__file__).resolve().parent
CSRC = PKG / "csrc"
OBJ = PKG / "build"
LIB = PKG / "libzipage_b200.so"
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-O3", "-lineinfo", "-std=c++17",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr",
] + os.environ.get("ZIPAGE_NVCC_FLAGS", "").split()

# sources of one model family (stems of csrc/*.cu)
PARTS = {
    "similorn": ("zp_api", "zp_host_sched", "zp_mlstm", "zp_mlstm_chunk", "zp_mlstm_tc", "zp_rows", "zp_step", "zp_tc",
                 "zp_window_attn", "zp_window_attn_mma", "zp_window_attn_tc"),
    "dobedra": ("zp_api", "zp_host_sched", "zp_latent", "zp_latent_decode_tc", "zp_latent_prefill_tc", "zp_moe", "zp_moe_tc", "zp_rows", "zp_step", "zp_tc",
                "zp_window_attn", "zp_window_attn_mma", "zp_window_attn_tc"),
    "tukarax": ("zp_api", "zp_conv", "zp_delta", "zp_delta_tc", "zp_host_sched", "zp_moe", "zp_moe_tc", "zp_rope", "zp_rows", "zp_step", "zp_tc",
                "zp_window_attn", "zp_window_attn_mma", "zp_window_attn_tc"),
    "dinatar": ("zp_api", "zp_conv", "zp_host_sched", "zp_linear_state", "zp_linear_state_tc", "zp_moe", "zp_moe_tc", "zp_rows",
                "zp_step", "zp_tc", "zp_window_attn", "zp_window_attn_mma", "zp_window_attn_tc"),
}


def _headers():
    return sorted(CSRC.glob("*.cuh")) + sorted((PKG.parent / "include").glob("*.h"))


def _newest_header() -> float:
    return max(h.stat().st_mtime for h in _headers())


def _sources(part=None):
    return sorted(CSRC.glob("*.cu")) if part is None else [CSRC / f"{n}.cu" for n in PARTS[part]]


def _digest(part=None) -> str:
    """What a library was built from: flags, headers and sources by content."""
    h = hashlib.sha256(" ".join(FLAGS).encode())
    for f in _headers() + _sources(part):
        h.update(f.name.encode() + b"\0" + f.read_bytes())
    return h.hexdigest()


def library_path(part=None) -> Path:
    return LIB if part is None else PKG / f"libzipage_b200_{part}.so"


def _stamp(lib: Path) -> Path:
    return lib.with_suffix(".so.src")


def is_current(part=None) -> bool:
    lib = library_path(part)
    return lib.exists() and _stamp(lib).exists() and _stamp(lib).read_text() == _digest(part)


def ensure(part=None) -> Path:
    """A library that holds the family's kernels and is current with the sources, compiled if there
    is none; the bindings load it from here on."""
    if is_current():
        part = None
    elif not is_current(part):
        with open(PKG / ".build.lock", "w") as lock:
            fcntl.flock(lock, fcntl.LOCK_EX)
            if not is_current(part):
                build(part=part)
    from . import _hostlib, _lib
    _lib.LIB_PATH = _hostlib.LIB_PATH = library_path(part)
    return library_path(part)


def build(force: bool = False, verbose: bool = False, part=None) -> Path:
    OBJ.mkdir(exist_ok=True)
    srcs, lib = _sources(part), library_path(part)
    hdr_time = _newest_header()
    jobs = []
    for s in srcs:
        o = OBJ / (s.stem + ".o")
        if force or not o.exists() or o.stat().st_mtime < max(s.stat().st_mtime, hdr_time):
            cmd = [NVCC, *FLAGS, "-c", str(s), "-o", str(o)]
            if verbose:
                cmd.insert(1, "-Xptxas=-v")
            jobs.append(cmd)

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        return cmd, r

    with ThreadPoolExecutor(max_workers=min(8, max(1, len(jobs)))) as ex:
        for cmd, r in ex.map(run, jobs):
            if verbose or r.returncode:
                sys.stderr.write(" ".join(cmd) + "\n" + r.stdout + r.stderr)
            if r.returncode:
                raise RuntimeError(f"nvcc failed on {cmd[-3]}")
    objs = [str(OBJ / (s.stem + ".o")) for s in srcs]
    if jobs or not is_current(part):
        tmp = lib.with_suffix(f".so.{os.getpid()}")
        cmd = [NVCC, "-shared", "-o", str(tmp), *objs, "-lcudart"]
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode:
            sys.stderr.write(r.stdout + r.stderr)
            raise RuntimeError("link failed")
        os.replace(tmp, lib)
        _stamp(lib).write_text(_digest(part))
    return lib


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
