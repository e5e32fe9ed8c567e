"""In-tree build of libmonofab.so with nvcc for sm_100a.

`python -m monoserve_b200.build` (or `build()`) compiles the CUDA sources under
`monoserve_b200/csrc/` into `monoserve_b200/libmonofab.so`.  nvcc cross-compiles
without a GPU.  Objects are rebuilt only when a source or header is newer.
"""
import os
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "build")
LIB = os.path.join(HERE, "libmonofab.so")
SOURCES = ["api.cu", "moe_aux.cu", "expert_gemm.cu", "pack_static.cu", "fabric_device.cu", "fabric_layer_rows.cu", "fabric_layer_scan.cu", "fabric_layer_memory.cu", "fabric_layer_gated.cu", "fabric_layer_residual.cu", "fabric_layer_attention.cu", "fabric_layer_latent.cu", "fabric_layer_latent_mma.cu", "fabric_layer_latent_direct.cu", "fabric_host.cu", "attention.cu", "host_loop.cu", "ep_exchange.cu", "release.cu", "plan_model.cu", "plan_admission.cu", "plan_api.cu"]
NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr"]
# The fabric kernel calls the tiles of the fabric_layer_*.cu files across translation units.
RELOCATABLE = {s for s in SOURCES if s == "fabric_device.cu" or s.startswith("fabric_layer_")}


def _nvcc():
    for cand in (os.environ.get("NVCC"), "/usr/local/cuda/bin/nvcc", "nvcc"):
        if cand and (os.path.isabs(cand) and os.path.exists(cand) or not os.path.isabs(cand)):
            return cand
    raise RuntimeError("nvcc not found")


def _newest_header():
    t = 0.0
    for root in (CSRC, os.path.join(HERE, "..", "include")):
        for f in os.listdir(root):
            if f.endswith((".h", ".cuh")):
                t = max(t, os.path.getmtime(os.path.join(root, f)))
    return t


def build(verbose=False, force=False):
    os.makedirs(OBJ, exist_ok=True)
    nvcc = _nvcc()
    hdr_t = _newest_header()
    jobs = []
    for src in SOURCES:
        s = os.path.join(CSRC, src)
        o = os.path.join(OBJ, src.replace(".cu", ".o"))
        if force or not os.path.exists(o) or os.path.getmtime(o) < max(os.path.getmtime(s), hdr_t):
            cmd = [nvcc, *NVCC_FLAGS, *(["-rdc=true"] if src in RELOCATABLE else []), "-c", s, "-o", o]
            if verbose:
                cmd.insert(1, "-Xptxas=-v")
            jobs.append(cmd)

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError("nvcc failed:\n" + " ".join(cmd) + "\n" + r.stdout + r.stderr)
        return r.stderr

    with ThreadPoolExecutor(max_workers=8) as ex:
        logs = list(ex.map(run, jobs))
    if verbose:
        for log in logs:
            sys.stderr.write(log)
    objs = [os.path.join(OBJ, s.replace(".cu", ".o")) for s in SOURCES]
    if jobs or not os.path.exists(LIB):
        cmd = [nvcc, "-shared", "-o", LIB, *objs, "-gencode", "arch=compute_100a,code=sm_100a",
               "-Xcompiler", "-fPIC"]
        run(cmd)
    return LIB


if __name__ == "__main__":
    print(build(verbose="-v" in sys.argv, force="-f" in sys.argv))
