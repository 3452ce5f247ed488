"""Which CUDA sources a model has compiled: every entry point belongs to one source, a source's key follows the headers it
includes, and a model names the sources of its parts and no others."""
import ctypes
import re

import pytest
import torch

from llm_serving_engine_b200.csrc import build
from llm_serving_engine_b200.kernels import library


def test_every_declared_entry_point_belongs_to_one_source():
    owners = {}
    for path in build.sources():
        for name in set(build.exported_names(path)):
            assert name not in owners, f"{name} in {path.stem} and {owners[name]}"
            owners[name] = path.stem
    assert set(library._SIGNATURES) <= set(owners)


def test_declared_argument_types_are_those_of_the_sources():
    kinds = {"int": ctypes.c_int, "long long": ctypes.c_longlong, "float": ctypes.c_float, "unsigned": ctypes.c_uint,
             "unsigned int": ctypes.c_uint, "cudaStream_t": ctypes.c_void_p}
    checked = set()
    for path in build.sources():
        for name, arguments in re.findall(r'extern "C" int\s+(lse_\w+)\s*\(([^)]*)\)', path.read_text()):
            if name not in library._SIGNATURES:
                continue
            want = []
            for argument in re.sub(r"//[^\n]*", "", arguments).split(","):
                words = argument.split()
                if not words or words == ["void"]:
                    continue
                want.append(ctypes.c_void_p if "*" in argument else kinds[" ".join(words[:-1])])
            assert library._SIGNATURES[name] == want, name
            checked.add(name)
    assert checked == set(library._SIGNATURES)


def test_a_sources_key_follows_what_it_includes(tmp_path, monkeypatch):
    monkeypatch.setattr(build, "CSRC", tmp_path)
    (tmp_path / "inner.cuh").write_text("int inner;\n")
    (tmp_path / "outer.cuh").write_text('#include "inner.cuh"\n')
    (tmp_path / "a.cu").write_text('#include "outer.cuh"\n')
    (tmp_path / "b.cu").write_text("int b;\n")
    before = [build._key(tmp_path / name, ["-O3"]) for name in ("a.cu", "b.cu")]
    (tmp_path / "inner.cuh").write_text("int other;\n")
    after = [build._key(tmp_path / name, ["-O3"]) for name in ("a.cu", "b.cu")]
    assert after[0] != before[0] and after[1] == before[1]
    assert build._key(tmp_path / "b.cu", ["-O2"]) != after[1]


def test_an_unknown_source_is_an_error():
    with pytest.raises(build.BuildError, match="no CUDA source"):
        build.library_paths(["no_such_source"], verbose=False)


def test_a_model_names_the_sources_of_its_parts_only():
    from llm_serving_engine_b200.cli import RANDOM_MODELS, tiny_config
    from llm_serving_engine_b200.config import load_config
    from llm_serving_engine_b200.models.decoder import kernel_sources

    known = {path.stem for path in build.sources()}
    needed = {}
    for name in RANDOM_MODELS:
        _, _, spec = load_config(tiny_config(name=name))
        for dtype in (torch.float32, torch.bfloat16):
            sources = kernel_sources(spec, dtype)
            assert sources <= known
            assert ("gemm_f32" in sources) == (dtype == torch.float32) and ("gemm_tcgen05" in sources) == (dtype == torch.bfloat16)
            needed[name] = sources
    assert "delta_memory" in needed["kofipel"] and "delta_memory" not in needed["sebudra"]
    assert {"selective_scan", "short_conv", "mlstm", "tanh_norm"} <= needed["tufevik"]
    assert "elementwise" in needed["givelix"] and "residual_streams" in needed["givelix"] and "moe" not in needed["givelix"]


def test_libraries_share_the_switch_of_dependent_launches():
    """Two libraries in one process have one switch: built here (nvcc needs no GPU), loaded, compared by address."""
    paths = build.library_paths(["elementwise", "tanh_norm"], verbose=False)
    places = {ctypes.addressof(ctypes.c_int.in_dll(ctypes.CDLL(str(path)), "lse_pdl_enabled")) for path in paths.values()}
    assert len(places) == 1
