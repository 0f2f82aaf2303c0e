"""Compile csrc/*.cu for sm_100a into lib/libferrite_b200.so with nvcc (in-tree, no JIT cache).

    python -m ferrite_b200.build            # build if sources are newer than the library
    python -m ferrite_b200.build --force

A checkout that has no library yet and is asked to run one model compiles what that model's family needs (FAMILY_SOURCES);
the library then says so (lib/sources.txt), and a full build, or another family's, adds the rest.
"""
import concurrent.futures
import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
SRC = os.path.join(HERE, "csrc")
OBJ = os.path.join(HERE, "build")
LIB = os.path.join(HERE, "lib", "libferrite_b200.so")
NVCC = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "-Xcompiler", "-fPIC",
         "-Xptxas", "-v"]


# what a family runs on where that is a part of the whole: its kernels, the sampling head, the general operators
FAMILY_SOURCES = {"binutar": ["api.cu", "decode_misc.cu", "dense.cu", "generic.cu", "latent.cu", "latent_tcgen05.cu", "recurrent.cu", "router.cu", "selective_prompt.cu"],
                  "labepel": ["api.cu", "decode_misc.cu", "dense.cu", "experts.cu", "generic.cu", "heads_attention.cu", *(f"heads_attention_{n}.cu" for n in (64, 128, 192, 256)), "heads_prompt.cu", "router.cu", "rows.cu"]}
FAMILY_SOURCES["vunadra"] = sorted({*FAMILY_SOURCES["labepel"], "latent.cu", "latent_tcgen05.cu"})
FAMILY_SOURCES["ronavik"] = sorted({*FAMILY_SOURCES["labepel"], "recurrent.cu", "selective_prompt.cu", "short_conv.cu"})
LINKED = os.path.join(HERE, "lib", "sources.txt")  # the sources a part of a library holds (no such file: all of them)


def sources():
    return sorted(f for f in os.listdir(SRC) if f.endswith(".cu"))


def linked():
    """The sources the library holds."""
    if not os.path.exists(LINKED):
        return sources()
    with open(LINKED) as f:
        return f.read().split()


def ensure(family, mode="bf16"):
    """Build what a model of this family needs in this precision, unless it is there (block floats: the whole library)."""
    need = FAMILY_SOURCES.get(family) if mode in ("bf16", "fp32") else None
    return build(only=need)


def stale(need=None):
    if not os.path.exists(LIB) or not set(need or sources()) <= set(linked()):
        return True
    built = os.path.getmtime(LIB)
    deps = [os.path.join(SRC, f) for f in os.listdir(SRC)] + [os.path.join(HERE, "..", "include", "ferrite_b200.h")]
    return any(os.path.getmtime(d) > built for d in deps)


def compile_one(name):
    obj = os.path.join(OBJ, name[:-3] + ".o")
    hdrs = [os.path.join(SRC, f) for f in os.listdir(SRC) if f.endswith((".cuh", ".h"))] + [os.path.join(HERE, "..", "include", "ferrite_b200.h")]
    newest = max(os.path.getmtime(p) for p in [os.path.join(SRC, name)] + hdrs)
    if os.path.exists(obj) and os.path.getmtime(obj) > newest:
        return name, ""
    r = subprocess.run([NVCC, *FLAGS, "-c", os.path.join(SRC, name), "-o", obj], capture_output=True, text=True)
    if r.returncode:
        raise RuntimeError(f"nvcc failed on {name}:\n{r.stdout}\n{r.stderr}")
    return name, r.stderr


def build(force=False, verbose=False, only=None):
    """only: some of the sources; what an existing library holds besides is kept."""
    if not force and not stale(only):
        return LIB
    names = sources() if only is None else sorted(set(only) | (set(linked()) if os.path.exists(LIB) else set()))
    os.makedirs(OBJ, exist_ok=True)
    os.makedirs(os.path.dirname(LIB), exist_ok=True)
    with concurrent.futures.ThreadPoolExecutor(max_workers=os.cpu_count() or 4) as pool:
        logs = list(pool.map(compile_one, names))
    if verbose:
        for name, log in logs:
            print(f"== {name}\n{log}")
    objs = [os.path.join(OBJ, f[:-3] + ".o") for f in names]
    r = subprocess.run([NVCC, "-shared", "-o", LIB, *objs, "-gencode", "arch=compute_100a,code=sm_100a"], capture_output=True, text=True)
    if r.returncode:
        raise RuntimeError(f"link failed:\n{r.stdout}\n{r.stderr}")
    if names != sources():
        with open(LINKED, "w") as f:
            f.write("\n".join(names) + "\n")
    elif os.path.exists(LINKED):
        os.remove(LINKED)
    return LIB


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
