"""Compile the CUDA sources in ``based_b200/csrc`` into one C-ABI shared library (sm_100a)."""
import glob
import os
import shutil
import subprocess

PKG = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(PKG)
CSRC = os.path.join(PKG, "csrc")
LIBDIR = os.path.join(PKG, "_lib")
LIBNAME = "libbased_b200.so"
# Sources of libraries for the hybrid stacks and for the post-norm stacks alone.  capi.cu refers to the other kernels weakly:
# in such a library their entry points answer BASED_ERR_IMPL.
HYBRID = ("capi.cu", "norm_act.cu", "decode_linear.cu", "short_conv.cu", "gated_delta.cu", "gated_delta_chunk.cu", "rglru.cu",
          "rglru_tc.cu", "latent_attention.cu", "latent_decode.cu", "latent_prefill_tc.cu")
POSTNORM = ("capi.cu", "norm_act.cu", "decode_linear.cu", "latent_attention.cu", "tied_attention.cu", "tied_decode.cu",
            "tied_prefill_tc.cu", "lightning.cu", "lightning_tc.cu", "token_side.cu")
PARTS = {"hybrid": ("libbased_b200_hybrid.so", HYBRID), "postnorm": ("libbased_b200_postnorm.so", POSTNORM)}
_chosen = None   # library of the part this process asked for, when that is not the whole one

def library_path() -> str:
    """Path of the shared library; the environment variable BASED_B200_LIB overrides it."""
    return os.environ.get("BASED_B200_LIB") or _chosen or os.path.join(LIBDIR, LIBNAME)


def _sources(part=None):
    if part is not None:
        return [os.path.join(CSRC, name) for name in PARTS[part][1]]
    return sorted(glob.glob(os.path.join(CSRC, "*.cu")))


def _stale(lib: str) -> bool:
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    deps = _sources() + glob.glob(os.path.join(CSRC, "*.cuh")) + glob.glob(os.path.join(ROOT, "include", "*.h"))
    return any(os.path.getmtime(d) > t for d in deps)


def build_library(force: bool = False, verbose: bool = False, part: str = None) -> str:
    """Build (if stale) and return the path of the shared library.  Needs ``nvcc`` only; no GPU.  ``part`` names a subset
    of the kernels that is enough for the caller: only those are compiled, unless the whole library is there already."""
    global _chosen
    if os.environ.get("BASED_B200_LIB"):
        return library_path()  # an explicitly chosen library is used as it is
    lib = os.path.join(LIBDIR, LIBNAME)
    if not force and not _stale(lib):
        _chosen = None
        return lib
    if part is not None:
        lib = _chosen = os.path.join(LIBDIR, PARTS[part][0])
        if not force and not _stale(lib):
            return lib
    else:
        _chosen = None
    nvcc = shutil.which("nvcc") or "/usr/local/cuda/bin/nvcc"
    if not os.path.exists(nvcc):
        raise RuntimeError("nvcc not found: cannot build libbased_b200.so")
    os.makedirs(LIBDIR, exist_ok=True)
    objs = []
    procs = []
    objdir = os.path.join(LIBDIR, "obj")
    os.makedirs(objdir, exist_ok=True)
    for src in _sources(part):
        obj = os.path.join(objdir, os.path.basename(src)[:-3] + ".o")
        objs.append(obj)
        cmd = [nvcc, "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
               "-Xcompiler", "-fPIC", "-I" + os.path.join(ROOT, "include"), "-I" + CSRC, "-c", src, "-o", obj]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
    for src, p in procs:
        out, _ = p.communicate()
        if verbose and out:
            print(out)
        if p.returncode != 0:
            raise RuntimeError(f"nvcc failed on {src}:\n{out}")
    link = [nvcc, "-gencode", "arch=compute_100a,code=sm_100a", "-Xcompiler", "-fPIC", "-shared", "-o", lib + ".new"] + objs
    r = subprocess.run(link, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"link failed:\n{r.stdout}")
    os.replace(lib + ".new", lib)
    return lib


if __name__ == "__main__":
    import sys
    print(build_library(force="--force" in sys.argv, verbose="-v" in sys.argv))
