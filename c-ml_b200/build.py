"""Builds lib/libcml_b200.so: every csrc/*.cu with nvcc for sm_100a, every csrc/*.c and
host/*.c with gcc -std=c11, linked into one shared library that exports the cmlb200 C-ABI
and the C-ML-compatible host API -- exactly the functions and variables the two public headers
declare (a linker version script generated from include/*.h hides everything else).
Incremental (mtime based). No GPU is needed to build.

The programs under programs/ become executables in lib/. cml_generate links the library's objects; trace_run
links only what a model folder needs, so that a fresh checkout compiles a few files.

  build.py [-v] [--program NAME]"""
import os
import re
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

PKG = Path(__file__).resolve().parent
ROOT = PKG.parent
OBJ = PKG / "lib" / "obj"
LIB = PKG / "lib" / "libcml_b200.so"

NVCC_FLAGS = ["-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17",
              "-Xcompiler", "-fPIC", "-Xcompiler", "-fvisibility=default"]
CC_FLAGS = ["-std=c11", "-O2", "-fPIC", "-Wall", "-Wextra", "-D_POSIX_C_SOURCE=200809L"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found; the CUDA extension cannot be built")


def _headers():
    return list((ROOT / "include").glob("*.h")) + list((PKG / "csrc").glob("*.cuh")) + list((PKG / "host").glob("*.h"))


def _stale(out: Path, deps) -> bool:
    if not out.exists():
        return True
    t = out.stat().st_mtime
    return any(Path(d).stat().st_mtime > t for d in deps)


def _compile(src: Path, verbose: bool):
    obj = OBJ / (src.parent.name + "_" + src.stem + ".o")
    if not _stale(obj, [src] + _headers()):
        return obj, None
    inc = ["-I", str(ROOT / "include"), "-I", str(PKG / "csrc"), "-I", str(PKG / "host")]
    if src.suffix == ".cu":
        cmd = [_nvcc()] + NVCC_FLAGS + (["-Xptxas", "-v"] if verbose else []) + inc + ["-c", str(src), "-o", str(obj)]
    else:
        cmd = [os.environ.get("CC", "gcc")] + CC_FLAGS + inc + ["-I", "/usr/local/cuda/include", "-c", str(src), "-o", str(obj)]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"compile failed: {' '.join(cmd)}\n{r.stdout}\n{r.stderr}")
    return obj, (r.stdout + r.stderr)


def public_symbols():
    """Names the public headers declare: every function prototype and every `extern` variable."""
    names = set()
    for h in sorted((ROOT / "include").glob("*.h")):
        text = re.sub(r"/\*.*?\*/", "", h.read_text(), flags=re.S)
        text = re.sub(r"//[^\n]*", "", text)
        for m in re.finditer(r"\b([A-Za-z_][A-Za-z0-9_]*)\s*\([^;{}()]*(?:\([^()]*\)[^;{}()]*)*\)\s*;", text):
            if m.group(1) not in ("defined", "sizeof", "__attribute__"):
                names.add(m.group(1))
        for m in re.finditer(r"\bextern\s+(?!\"C\")[^;()]*?\b([A-Za-z_][A-Za-z0-9_]*)\s*(?:\[[^\]]*\])?\s*;", text):
            names.add(m.group(1))
    return sorted(names)


def _version_script() -> Path:
    path = OBJ / "exports.map"
    body = "{\n  global:\n" + "".join(f"    {n};\n" for n in public_symbols()) + "  local: *;\n};\n"
    if not path.exists() or path.read_text() != body:
        path.write_text(body)
    return path


# Sources of the programs besides their own; None: everything the library holds.
PROGRAMS = {
    "trace_run": ["host/cml_json.c", "host/cml_safetensors.c", "host/cml_lm.c", "host/cml_lm_layered.c", "host/cml_lm_delta.c", "host/cml_lm_gru.c", "host/cml_lm_talk.c", "host/cml_paged.c", "host/cml_serving.c",
                  "host/cml_sampling.c", "host/cml_tensor.c", "host/cml_tokenizer.c", "csrc/shim.cu", "csrc/argmax.cu",
                  "csrc/lm_rows.cu", "csrc/attention_rows.cu", "csrc/latent_rows.cu", "csrc/attention_latent.cu", "csrc/attention_latent_tc.cu", "csrc/moe_rows.cu", "csrc/delta_rule.cu", "csrc/gru_rows.cu", "csrc/rotate_rows.cu", "csrc/talk_scores.cu", "csrc/gemv_bf16.cu", "csrc/gemm_bf16.cu", "csrc/llm_ops_f32.cu", "csrc/paged_attention.cu"],
    "cml_generate": None,
}
LINK_LIBS = ["-lcudart_static", "-ldl", "-lpthread", "-lrt", "-lm"]


def _library_sources():
    return sorted((PKG / "csrc").glob("*.cu")) + sorted((PKG / "csrc").glob("*.c")) + sorted((PKG / "host").glob("*.c"))


def _compile_all(srcs, verbose):
    OBJ.mkdir(parents=True, exist_ok=True)
    with ThreadPoolExecutor(max_workers=min(8, len(srcs))) as ex:
        results = list(ex.map(lambda s: _compile(s, verbose), srcs))
    for _, log in results:
        if verbose and log:
            print(log)
    return [o for o, _ in results]


def _link(cmd):
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError(f"link failed: {' '.join(cmd)}\n{r.stdout}\n{r.stderr}")


def build(verbose: bool = False) -> Path:
    objs = _compile_all(_library_sources(), verbose)
    vs = _version_script()
    if _stale(LIB, objs + [vs]):
        _link([_nvcc(), "-shared", "-o", str(LIB)] + [str(o) for o in objs] + ["-Xlinker", "-Bsymbolic", "-Xlinker", f"--version-script={vs}"] + LINK_LIBS)
    return LIB


def build_program(name: str, verbose: bool = False) -> Path:
    srcs = PROGRAMS[name]
    objs = _compile_all([PKG / "programs" / f"{name}.c"] + (_library_sources() if srcs is None else [PKG / s for s in srcs]), verbose)
    out = PKG / "lib" / name
    if _stale(out, objs):
        _link([_nvcc(), "-o", str(out)] + [str(o) for o in objs] + LINK_LIBS)
    return out


if __name__ == "__main__":
    v = "-v" in sys.argv
    if "--program" in sys.argv:
        print(build_program(sys.argv[sys.argv.index("--program") + 1], v))
    else:
        print(build(v))
