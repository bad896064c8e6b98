"""Which CUDA sources a model's first call compiles (no GPU): every kernel that a part can reach through the kernel
library lies in the core sources or in one the part names, and the libraries of chosen sources are named, stamped and
linked apart from the library of all sources."""
import inspect
import os
import re

import pytest

import tffinfer_b200.models  # noqa: F401  registers the architectures
import tffinfer_b200.parts  # noqa: F401  registers the parts
from tffinfer_b200 import registry
from tffinfer_b200.csrc import build
from tffinfer_b200.kernels.library import CudaKernels
from tffinfer_b200.parts.moe import RoutedExperts


def _file_of_symbol():
    out = {}
    for src in build.sources():
        with open(os.path.join(build.CSRC_DIR, src)) as f:
            for name in re.findall(r"TFF_API [a-z ]+\**\s?(tff_\w+)", f.read()):
                out[name] = src[:-3]
    return out


def _symbols_of_methods():
    """Method of the kernel library -> entry points it can reach, through the methods it calls too."""
    direct, calls = {}, {}
    for name, fn in inspect.getmembers(CudaKernels, callable):
        if name.startswith("__"):
            continue
        try:
            text = inspect.getsource(fn)
        except (TypeError, OSError):
            continue
        direct[name] = set(re.findall(r"self\.lib\.(tff_\w+)", text))
        calls[name] = set(re.findall(r"self\.(\w+)\(", text))
    changed = True
    while changed:
        changed = False
        for name in direct:
            for other in calls[name]:
                if other in direct and not direct[other] <= direct[name]:
                    direct[name] |= direct[other]
                    changed = True
    return direct


# what a method reaches only for parts that ask for it in other words than by calling the method
SPARED = {"routed_experts": {"gemm_tc_cluster"}}      # a gated shared expert: named by the instance


@pytest.mark.parametrize("family", registry.PART_FAMILIES)
def test_parts_name_the_sources_of_the_kernels_they_can_reach(family):
    where, reach = _file_of_symbol(), _symbols_of_methods()
    assert len(where) > 50 and reach["latent_attend"] > {"tff_latent_finish", "tff_attention_tile", "tff_gemm_grouped_mma"}
    for kind in registry.registered_parts(family):
        cls = registry.get_part(family, kind)
        if not cls.__module__.startswith("tffinfer_b200."):
            continue                                   # registered by another test
        text = "".join(inspect.getsource(c) for c in cls.__mro__ if c.__module__.startswith("tffinfer_b200."))
        used = {m for m in re.findall(r"\bops\.(\w+)", text) if m in reach} | ({"rmsnorm_pair"} if "rmsnorm_pair" in text else set())
        files = {where[s] for m in used for s in reach[m]} - set(build.CORE)
        if family in ("block", "connector"):
            files -= {"streams"}                       # a model of several streams names it itself
        if kind == "parallel":
            continue                                   # what its branches name
        part = object.__new__(cls)
        part.gated, part.shared_intermediate = True, 0
        named = set(part.kernel_files()) if hasattr(cls, "kernel_files") else set()
        assert files - SPARED.get(kind, set()) <= named, f"{family} '{kind}' reaches {sorted(files - named)}"


def test_a_gated_shared_expert_names_its_product():
    make = lambda **kw: set(RoutedExperts(16, 16, 2, 1, **kw).kernel_files())
    assert "gemm_tc_cluster" in make(shared_intermediate=16) and "gemm_tc_cluster" not in make()
    assert "gemm_tc_cluster" not in make(shared_intermediate=16, gated=False, activation="relu2")


def test_chosen_sources_and_library_names(tmp_path, monkeypatch):
    monkeypatch.setenv("TFFINFER_BUILD_DIR", str(tmp_path))
    assert build.chosen_sources(None) == build.sources()
    some = build.chosen_sources(["latent", "moe", "latent"])
    assert some == sorted({f + ".cu" for f in build.CORE + ("latent", "moe")})
    with pytest.raises(RuntimeError):
        build.chosen_sources(["no_such_file"])
    seen = []

    def fake_compile(bdir, verbose=True, extra_flags=None, srcs=None, lib_name=build.LIB_NAME):
        seen.append((lib_name, srcs))
        open(os.path.join(bdir, lib_name), "w").close()
        return os.path.join(bdir, lib_name)
    monkeypatch.setattr(build, "compile_all", fake_compile)
    a = build.library_path(files=["latent"])
    assert build.library_path(files=["latent"]) == a and len(seen) == 1          # up to date: nothing is compiled
    b = build.library_path(files=["moe"])
    assert a != b and len(seen) == 2 and "latent.cu" in seen[0][1] and "latent.cu" not in seen[1][1]
    full = build.library_path()
    assert os.path.basename(full) == build.LIB_NAME and seen[2][1] == build.sources()
    assert build.library_path(files=["latent"]) == full and len(seen) == 3       # the library of all sources serves
