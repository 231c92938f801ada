"""Calls into the kernel library go through ctypes, which accepts surplus arguments silently: every registration agrees with the C
declaration, and every call passes as many arguments as were registered."""
import ast
import re
from pathlib import Path

PACKAGE = Path(__file__).resolve().parent.parent / "eredu_b200"
KINDS = {"P": "P", "I": "I", "L": "I", "F": "F"}


def registered():
    """Entry point -> argument kinds, from ``native.register(name, result, kinds)``."""
    out = {}
    for path in sorted((PACKAGE / "ops").glob("*.py")):
        for node in ast.walk(ast.parse(path.read_text())):
            if isinstance(node, ast.Call) and getattr(node.func, "attr", "") == "register" and len(node.args) == 3:
                kinds = eval(compile(ast.Expression(node.args[2]), str(path), "eval"), {**KINDS, "native": type("N", (), KINDS)})
                out[node.args[0].value] = "".join(kinds)
    return out


def declared():
    """Entry point -> argument kinds of the C declaration (long long counts as an integer)."""
    out = {}
    for path in sorted((PACKAGE / "csrc").rglob("*.cu")):
        for name, args in re.findall(r'extern "C"\s+[\w ]+?\s(eredu_\w+)\(([^)]*)\)\s*\{', path.read_text()):
            parts = [a.strip() for a in args.replace("\n", " ").split(",") if a.strip()]
            out[name] = "".join("P" if "*" in a or "cudaStream_t" in a else "F" if a.startswith("float ") else "I" for a in parts)
    return out


def test_registrations_agree_with_the_declarations():
    c, py = declared(), registered()
    assert len(py) > 20
    for name, kinds in py.items():
        assert name in c and c[name] == kinds, (name, kinds, c.get(name))


def test_calls_pass_what_is_registered():
    py, seen = registered(), 0
    for path in sorted(PACKAGE.rglob("*.py")):
        for node in ast.walk(ast.parse(path.read_text())):
            name = getattr(getattr(node, "func", None), "attr", "")
            if isinstance(node, ast.Call) and name in py and not any(isinstance(a, ast.Starred) for a in node.args):
                assert len(node.args) == len(py[name]), (path.name, node.lineno, name)
                seen += 1
    assert seen > 20
