"""The ctypes prototypes and argument blocks of ``kernels/ops.py`` against the C sources, without a GPU: a prototype with too
few arguments would pass a pointer as a 32-bit number, a block with a missing field would shift all that follow."""
import ctypes
import glob
import importlib
import os
import re

ops = importlib.import_module("daisi-llogos_b200.kernels.ops")
CSRC = os.path.join(os.path.dirname(ops.__file__), "..", "csrc")

C_SIZES = {"int": 4, "float": 4, "long long": 8, "unsigned long long": 8}


def _text(path):
    with open(path) as f:
        return re.sub(r"//[^\n]*", "", f.read())


def test_every_entry_point_has_a_prototype_of_its_length():
    with open(ops.__file__) as f:
        src = f.read()
    protos = {m.group(1): len([x for x in m.group(2).split(",") if x.strip()])
              for m in re.finditer(r"lib\.(llg_\w+)\.argtypes = \[(.*?)\]", src, re.S)}
    seen = 0
    for path in glob.glob(os.path.join(CSRC, "*.cu")):
        for m in re.finditer(r"LLG_API\s+[\w ]+?\s*\*?(llg_\w+)\(([^)]*)\)\s*\{", _text(path)):
            args = [x for x in m.group(2).split(",") if x.strip()]
            if m.group(1) in protos:
                seen += 1
                assert protos[m.group(1)] == len(args), (os.path.basename(path), m.group(1), len(args), protos[m.group(1)])
    assert seen > 40


def _c_struct(text, name, known):
    """``[(field, size)]`` of a plain C structure."""
    body = re.search(r"struct %s \{(.*?)\n\};" % name, text, re.S).group(1)
    defines = {k: int(v) for k, v in re.findall(r"#define (LLG_\w+) (\d+)\s", text)}
    fields = []
    for decl in body.split(";"):
        decl = " ".join(decl.split())
        if not decl:
            continue
        m = re.match(r"(?:const )?((?:unsigned )?long long|\w+)\s*(.*)$", decl)
        for var in m.group(2).split(","):
            var = var.strip()
            count = re.search(r"\[(\w+)\]", var)
            times = 1 if count is None else int(defines.get(count.group(1), count.group(1)))
            size = 8 if "*" in var else known.get(m.group(1)) or C_SIZES[m.group(1)]
            fields.append((re.sub(r"\[.*\]|\*", "", var).strip(), size * times))
    return fields


def test_argument_blocks_have_the_fields_of_their_structures():
    text = _text(os.path.join(CSRC, "kernel_args.h"))
    known = {}
    names = [n[1:] for n, c in vars(ops).items() if isinstance(c, type) and issubclass(c, ctypes.Structure) and n.startswith("_")]
    found = [n for n in re.findall(r"\nstruct (\w+) \{", text) if n in names]
    assert len(found) >= 15
    for n in found:
        block = getattr(ops, "_" + n)
        want = _c_struct(text, n, known)
        got = [(f, ctypes.sizeof(t)) for f, t in block._fields_]
        assert got == want, n
        known[n] = ctypes.sizeof(block)
