"""Makes the package importable from a source checkout, compiling the kernel library if it is missing or
older than its sources."""
import importlib.util
import sys
from pathlib import Path

ROOT = Path(__file__).resolve().parent.parent


def load_package():
    spec = importlib.util.spec_from_file_location("_b200_build", ROOT / "sglang.cpp_b200" / "build.py")
    build = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(build)
    build.ensure_built()
    sys.path.insert(0, str(ROOT))
    import __graft_entry__

    return __graft_entry__.load_package()
