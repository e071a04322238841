"""The argument lists that ``ops/_lib.py`` declares for the kernel library are those of the C functions in ``csrc``: an argument
too many would be passed as a 32-bit int, whatever it is."""

import ctypes
import glob
import os
import re

from slime_b200.ops import _lib

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _kind(param: str):
    words = param.replace("*", " * ").split()
    if "*" in words or "cudaStream_t" in words:
        return ctypes.c_void_p
    for name, kind in (("float", ctypes.c_float), ("long", ctypes.c_long), ("unsigned", ctypes.c_uint), ("int", ctypes.c_int)):
        if name in words:
            return kind
    raise ValueError(param)


def test_declared_argument_lists_match_the_sources():
    found = {}
    for path in glob.glob(os.path.join(ROOT, "csrc", "*.cu")):
        text = re.sub(r"//[^\n]*", "", open(path).read())
        for name, params in re.findall(r'extern "C" (?:int|void) (sb_\w+)\(([^)]*)\)\s*\{', text):
            found[name] = [_kind(p) for p in params.split(",") if p.strip() and p.strip() != "void"]
    missing = [n for n in _lib._SIGS if n not in found]
    assert not missing, missing
    wrong = {n: (len(found[n]), len(a)) for n, a in _lib._SIGS.items() if list(a) != found[n]}
    assert not wrong, wrong
