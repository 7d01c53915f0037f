"""Test infrastructure: builds the 32-bit residual-stream kernel files (lp_linear.cu, lp_stream32.cu, lp_seqmix.cu, lp_winattn.cu, lp_mingru.cu, lp_mlstm.cu, lp_gla.cu, lp_moe.cu — kernels
AND their host entry points) for the CPU emulator: includes dropped, dynamic shared memory turned into a static buffer, launches
rewritten (launch_rewrite.py), runtime names from host_emu.h.  The result exports the same C symbols as the native library."""
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

ROOT = Path(__file__).resolve().parents[2]
SOURCES = ("lp_linear", "lp_stream32", "lp_seqmix", "lp_winattn", "lp_mingru", "lp_mlstm", "lp_gla", "lp_moe")


def build_emulated(out: Path) -> Path:
    sys.path.insert(0, str(ROOT / "tests/emu"))
    from launch_rewrite import rewrite_launches
    out.mkdir(parents=True, exist_ok=True)
    units = []
    for name in SOURCES:
        src = (ROOT / "leopard_b200/csrc" / f"{name}.cu").read_text()
        src = src.replace('#include <cuda_pipeline.h>\n', "")
        for line in ('#include "lp_host.h"\n', '#include "../../include/leopard_b200.h"\n'):
            assert line in src, (name, line)
            src = src.replace(line, "")
        src = src.replace("  extern __shared__ float dyn_smem[];", "  static float dyn_smem[1 << 16];")
        assert "extern __shared__" not in src and "asm" not in src, name
        src = rewrite_launches(src)
        assert "<<<" not in src, name
        (out / f"{name}_src.inc").write_text(src)
        unit = out / f"{name}_emu.cpp"
        unit.write_text('#include "host_emu.h"\n#include "leopard_b200.h"\n'
                        f'#include "{name}_src.inc"\n')
        units.append(str(unit))
    (out / "common_emu.cpp").write_text(
        '#include "host_emu.h"\nextern "C" {\nconst char* lp_last_error(void) { return lp::g_emu_err; }\n'
        'long long lp_launch_count(void) { return 0; }\nint lp_abi_version(void) { return 3; }\n}\n')
    lib = out / "libstream32_emu.so"
    # no unique symbols: the process may hold other emulated libraries, whose contexts of the same name have the threaded form
    flags = ["-fno-gnu-unique", "-std=c++20", "-O2", "-pthread", "-fPIC", "-ffp-contract=off", "-fno-strict-aliasing", "-DEMU_FIBERS", "-U_FORTIFY_SOURCE",
             "-I", str(out), "-I", str(ROOT / "tests/emu"), "-I", str(ROOT / "include")]

    def run(cmd):
        r = subprocess.run(cmd, capture_output=True, text=True)
        if r.returncode != 0:
            raise RuntimeError(r.stderr[-6000:])

    units.append(str(out / "common_emu.cpp"))
    with ThreadPoolExecutor(max_workers=8) as ex:
        list(ex.map(lambda u: run(["g++", *flags, "-c", u, "-o", u.replace(".cpp", ".o")]), units))
    run(["g++", "-shared", "-pthread", *[u.replace(".cpp", ".o") for u in units], "-o", str(lib)])
    return lib
