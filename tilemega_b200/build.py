"""Build libtilemega_b200.so in-tree with nvcc for sm_100a.

The library is the product: nothing in the package falls back to another
implementation when it is missing.
"""
from __future__ import annotations

import os
import shutil
import subprocess
from pathlib import Path

ROOT = Path(__file__).resolve().parent
CSRC = ROOT / "csrc"
LIB_DIR = ROOT / "lib"
LIBRARY = LIB_DIR / "libtilemega_b200.so"
# (object name, source, extra flags, components). The kernel source is compiled four times, side by side:
# plain (unsharded dense plans), extended (tensor parallelism, mixture of experts, QK norm), dense-batch
# (batch 16..64: GEMM stages on tcgen05 tiles) and e4m3 weights (the small-batch kernel with 8-bit weight pages).
# Component "all" is the whole library; "ragged" is what ragged plans need (seconds to build instead of minutes),
# with absent.cu in place of the other plan kinds.
COMPONENTS = ("all", "ragged")
ALL, BOTH = ("all",), COMPONENTS
UNITS = (("megakernel", "megakernel.cu", (), ALL), ("megakernel_extended", "megakernel.cu", ("-DTMB_EXTENDED=1",), ALL),
         ("megakernel_dense", "megakernel.cu", ("-DTMB_DENSE=1",), ALL), ("megakernel_fp8", "megakernel.cu", ("-DTMB_FP8=1",), ALL),
         ("runtime", "runtime.cu", (), BOTH), ("plan_spec", "plan_spec.cpp", (), BOTH), ("static_probe", "static_probe.cu", (), ALL),
         ("pack", "pack.cu", (), ALL), ("calibrate", "calibrate.cu", (), ALL), ("encoder", "encoder.cu", (), ALL),
         ("ragged", "ragged.cu", (), BOTH), ("ragged_spec", "ragged_spec.cpp", (), BOTH), ("linear", "linear.cu", (), BOTH),
         ("experts", "experts.cu", (), BOTH), ("mixers", "mixers.cu", (), BOTH), ("mixers_mma", "mixers_mma.cu", (), BOTH),
         ("latent", "latent.cu", (), BOTH), ("delta", "delta.cu", (), BOTH), ("delta_mma", "delta_mma.cu", (), BOTH), ("conv", "conv.cu", (), BOTH),
         ("rows", "rows.cu", (), BOTH), ("absent", "absent.cu", (), ("ragged",)))
# headers a source includes (directly or through another header): a unit is rebuilt when one of ITS headers changed
SPEC_HEADERS = ("plan_spec.h", "json.h", "params.h", "ragged_spec.h")
KERNEL_HEADERS = ("params.h", "ptx.cuh")
OP_HEADERS = ("ops.h", "ragged_limits.h", "element.cuh", "ptx.cuh", "tensor_map.h")
UNIT_HEADERS = {"megakernel.cu": KERNEL_HEADERS, "static_probe.cu": KERNEL_HEADERS, "calibrate.cu": ("ptx.cuh",), "pack.cu": (),
                "plan_spec.cpp": SPEC_HEADERS, "runtime.cu": SPEC_HEADERS + ("encoder.h", "ragged.h"),
                "encoder.cu": SPEC_HEADERS + ("encoder.h", "ptx.cuh", "tensor_map.h"), "absent.cu": SPEC_HEADERS + ("encoder.h",),
                "ragged_spec.cpp": SPEC_HEADERS + ("ragged_limits.h",), "ragged.cu": SPEC_HEADERS + OP_HEADERS + ("ragged.h",),
                "linear.cu": OP_HEADERS, "rows.cu": OP_HEADERS, "experts.cu": OP_HEADERS, "mixers.cu": OP_HEADERS + ("mixers.cuh",),
                "mixers_mma.cu": OP_HEADERS + ("mixers.cuh", "mma.cuh"), "latent.cu": OP_HEADERS + ("mixers.cuh", "mma.cuh"),
                "delta.cu": OP_HEADERS + ("mixers.cuh",), "delta_mma.cu": OP_HEADERS + ("mixers.cuh", "mma.cuh"), "conv.cu": OP_HEADERS}
SOURCES = tuple(sorted({unit[1] for unit in UNITS}))
HEADERS = tuple(sorted({header for headers in UNIT_HEADERS.values() for header in headers}))
ABI_HEADER = ROOT.parent / "include" / "tilemega_b200.h"


def library_path(component: str = "all") -> Path:
    return LIBRARY if component == "all" else LIB_DIR / f"libtilemega_b200_{component}.so"


def nvcc() -> str:
    found = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not Path(found).exists():
        raise RuntimeError("nvcc not found; the CUDA library cannot be built")
    return found


def _inputs(source: str) -> list[Path]:
    return [CSRC / name for name in (source,) + UNIT_HEADERS[source]] + [ABI_HEADER]


def _stale(component: str = "all") -> bool:
    library = library_path(component)
    if not library.exists():
        return True
    built = library.stat().st_mtime
    return any(path.stat().st_mtime > built for _, source, _, components in UNITS if component in components for path in _inputs(source))


def library_for(phase: str) -> Path:
    """The library a plan of this phase runs on: the whole one, unless only the ragged component is needed and the
    whole one has not been built (or is out of date)."""
    return build_library(component="ragged" if phase == "ragged" and _stale("all") else "all")


def build_library(force: bool = False, verbose: bool = False, component: str = "all") -> Path:
    """Compile the CUDA sources of a component into its library under lib/ (no GPU needed)."""
    library = library_path(component)
    if not force and not _stale(component):
        return library
    LIB_DIR.mkdir(exist_ok=True)
    objects = []
    common = ["-O3", "-std=c++17", "-Xcompiler", "-fPIC", "-gencode", "arch=compute_100a,code=sm_100a",
              "-lineinfo", "-diag-suppress", "177"]   # 177: helpers one of the kernel translation units does not use
    if verbose:
        common += ["-Xptxas", "-v"]
    build_dir = ROOT / "build"
    build_dir.mkdir(exist_ok=True)
    running = []
    for stem, name, flags, components in UNITS:
        if component not in components:
            continue
        obj = build_dir / (stem + ".o")
        objects.append(str(obj))
        if not force and not verbose and obj.exists() and all(path.stat().st_mtime <= obj.stat().st_mtime for path in _inputs(name)):
            continue   # this unit's object is newer than its source and every header
        cmd = [nvcc(), *common, *flags, "-x", "cu" if name.endswith(".cu") else "c++", "-c", str(CSRC / name), "-o",
               str(obj)]
        running.append((cmd, subprocess.Popen(cmd)))
    for cmd, process in running:
        if process.wait() != 0:
            raise subprocess.CalledProcessError(process.returncode, cmd)
    tmp = library.with_suffix(".so.tmp")
    subprocess.run([nvcc(), "-shared", "-o", str(tmp), *objects, "-gencode", "arch=compute_100a,code=sm_100a",
                    "-Xlinker", "--no-undefined", "-ldl"], check=True)
    os.replace(tmp, library)
    return library


if __name__ == "__main__":
    print(build_library(force=True, verbose=bool(os.environ.get("VERBOSE"))))
