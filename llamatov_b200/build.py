"""Compile the CUDA sources of the package into its shared libraries (sm_100a), in-tree:

  libllamatov_b200_common.so   errors, status word, launch counter, the small streaming operators
  libllamatov_b200.so          the Q8_0 path          (needs the common library)
  libllamatov_b200_dense.so    the bf16 / fp32 models (needs the common library)

Run as `python -m llamatov_b200.build [--group q8|dense] [--force] [-v]` or through `__graft_entry__.build()`.
A library is rebuilt when one of its sources is newer than it.
"""
import contextlib
import fcntl
import glob
import os
import subprocess
import sys
import tempfile

HERE = os.path.dirname(os.path.abspath(__file__))
CSRC = os.path.join(HERE, "csrc")
LIB = os.path.join(HERE, "libllamatov_b200.so")
COMMON_LIB = os.path.join(HERE, "libllamatov_b200_common.so")
DENSE_LIB = os.path.join(HERE, "libllamatov_b200_dense.so")
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
COMPILE = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC"]
_COMMON = ("lt_api.cu", "lt_elementwise.cu")
GROUPS = {"common": COMMON_LIB, "q8": LIB, "dense": DENSE_LIB}


def sources(group=None):
    """Sources of one library, or all of them."""
    out = []
    for src in sorted(glob.glob(os.path.join(CSRC, "*.cu"))):
        name = os.path.basename(src)
        g = "common" if name in _COMMON else ("dense" if name.startswith("lt_dn_") else "q8")
        if group is None or g == group:
            out.append(src)
    return out


def _stale(group):
    lib = GROUPS[group]
    if not os.path.exists(lib):
        return True
    t = os.path.getmtime(lib)
    deps = sources(group) + glob.glob(os.path.join(HERE, "..", "include", "*.h")) + [os.path.abspath(__file__)]
    deps += [h for h in glob.glob(os.path.join(CSRC, "*.cuh"))
             if group == "dense" or not os.path.basename(h).startswith("lt_dn_")]
    return any(os.path.getmtime(d) > t for d in deps)


@contextlib.contextmanager
def _lock(objdir):
    with open(os.path.join(objdir, ".lock"), "w") as f:
        fcntl.flock(f, fcntl.LOCK_EX)
        yield


def build(force=False, verbose=False, groups=("q8", "dense")):
    """Build the named libraries (and the common one) where a source is newer.  Returns the path of the last."""
    todo = ["common"] + [g for g in ("q8", "dense") if g in groups]
    if not force and not any(_stale(g) for g in todo):
        return GROUPS[todo[-1]]
    objdir = os.path.join(HERE, "build")
    os.makedirs(objdir, exist_ok=True)
    with _lock(objdir):
        todo_now = [g for g in todo if force or _stale(g)]
        procs = []
        for g in todo_now:
            for src in sources(g):
                obj = os.path.join(objdir, os.path.basename(src)[:-3] + ".o")
                cmd = [NVCC] + COMPILE + (["-Xptxas=-v"] if verbose else []) + ["-c", src, "-o", obj]
                procs.append((src, subprocess.Popen(cmd, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, text=True)))
        for src, p in procs:
            out, _ = p.communicate()
            if p.returncode != 0:
                raise RuntimeError("nvcc failed on %s:\n%s" % (src, out[-6000:]))
            if verbose and out:
                print(out)
        for g in todo_now:
            objs = [os.path.join(objdir, os.path.basename(s)[:-3] + ".o") for s in sources(g)]
            fd, tmp = tempfile.mkstemp(dir=objdir, suffix=".so")
            os.close(fd)
            link = [NVCC, "-shared", "-cudart", "shared", "-o", tmp] + objs
            if g != "common":
                link += ["-L", HERE, "-Xlinker", "--no-as-needed", "-Xlinker", "-l:" + os.path.basename(COMMON_LIB),
                         "-Xlinker", "-rpath=$ORIGIN"]
            else:
                link += ["-Xlinker", "-soname=" + os.path.basename(COMMON_LIB)]
            r = subprocess.run(link, capture_output=True, text=True)
            if r.returncode != 0:
                raise RuntimeError("link failed:\n%s" % r.stderr[-4000:])
            os.chmod(tmp, 0o755)
            os.replace(tmp, GROUPS[g])
    return GROUPS[todo[-1]]


if __name__ == "__main__":
    gs = [sys.argv[i + 1] for i, a in enumerate(sys.argv[:-1]) if a == "--group"] or ("q8", "dense")
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv, groups=gs))
