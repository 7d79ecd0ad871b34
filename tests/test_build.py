"""The kernel library builds for sm_100a without a GPU and exports its C entry points."""
import ctypes
import shutil

import pytest


@pytest.mark.skipif(shutil.which("nvcc") is None, reason="nvcc not installed")
def test_build_and_symbols():
    from ringattention_b200 import _build

    path = _build.build()
    assert path.exists()
    lib = ctypes.CDLL(str(path))
    for sym in ("ra_gemm_bf16", "ra_attn_fwd", "ra_attn_bwd", "ra_attn_bwd_prep", "ra_rmsnorm_fwd",
                "ra_rmsnorm_bwd", "ra_rope", "ra_swiglu_fwd", "ra_swiglu_bwd", "ra_xent_fwd_bwd",
                "ra_adamw", "ra_symm_barrier", "ra_peer_copy", "ra_last_error"):
        assert hasattr(lib, sym), sym
    flags = " ".join(_build.NVCC_FLAGS)
    assert "compute_100a" in flags and "sm_100a" in flags


@pytest.mark.skipif(shutil.which("nvcc") is None, reason="nvcc not installed")
@pytest.mark.parametrize("family", ["Dafelorn", "Kalonex", "Llama"])
def test_build_of_one_engines_sources(family, tmp_path, monkeypatch):
    """A library of only the sources an engine names exports what the engine calls and nothing of training."""
    from ringattention_b200 import _build
    from ringattention_b200.models import registry

    _build.build()
    monkeypatch.setattr(_build, "is_current", lambda: False)      # as in a fresh checkout; the objects are reused
    monkeypatch.setattr(_build, "LIB_PATH", tmp_path / "libpart.so")
    path = _build.build(only=registry.FAMILIES[family].sources)
    assert path.parent == tmp_path and path != _build.LIB_PATH
    lib = ctypes.CDLL(str(path))
    want = ["ra_last_error", "ra_decode_advance", "ra_small_m_linear", "ra_attn_fwd"]
    hybrid = ["ra_linear_f32", "ra_norm_f32", "ra_embed_f32", "ra_gemm_bf16_ex", "ra_small_m_linear_segments"]
    want += {"Dafelorn": hybrid + ["ra_attn_two_part", "ra_delta_step", "ra_delta_chunk_scan", "ra_latent_few_attend",
                                   "ra_latent_prep"],
             "Kalonex": hybrid + ["ra_attn_window", "ra_window_prep", "ra_window_attend", "ra_window_decode", "ra_moe_few",
                                  "ra_moe_route", "ra_moe_gemm", "ra_moe_combine", "ra_stream_pair", "ra_gated_act_f32",
                                  "ra_small_m_linear_gated", "ra_gemm_bf16_swiglu"],
             "Llama": ["ra_rmsnorm_fwd", "ra_rope_append", "ra_gemm_bf16_swiglu"]}[family]
    for sym in want:
        assert hasattr(lib, sym), sym
    for sym in ("ra_attn_bwd", "ra_adamw" if family != "Llama" else "ra_delta_step",
                "ra_moe_gemm" if family != "Kalonex" else "ra_latent_prep"):
        assert not hasattr(lib, sym), sym
    with pytest.raises(ValueError, match="no such sources"):
        _build.build(only=("nothing",))


@pytest.mark.skipif(shutil.which("nvcc") is None, reason="nvcc not installed")
def test_wheel_is_self_contained(tmp_path):
    """A wheel built from the tree, installed elsewhere, carries the kernel sources and the compiled library and
    loads it without the source tree."""
    import os
    import subprocess
    import sys

    src = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    # build from a copy, so that setuptools leaves its build/ and egg-info directories outside the repository
    # (the object files travel with the copy: nothing is recompiled)
    repo = str(tmp_path / "src")
    os.makedirs(repo)
    shutil.copytree(os.path.join(src, "ringattention_b200"), os.path.join(repo, "ringattention_b200"),
                    ignore=shutil.ignore_patterns("__pycache__"))
    for f in ("pyproject.toml", "setup.py", "README.md"):
        shutil.copy(os.path.join(src, f), repo)
    dist, site = tmp_path / "dist", tmp_path / "site"
    r = subprocess.run([sys.executable, "-m", "pip", "wheel", "--no-deps", "--no-build-isolation", "--no-index",
                        "-w", str(dist), repo], capture_output=True, text=True)
    assert r.returncode == 0, r.stdout + r.stderr
    whl = next(dist.glob("ringattention_b200-*.whl"))
    r = subprocess.run([sys.executable, "-m", "pip", "install", "--no-deps", "--no-index", "--target", str(site),
                        str(whl)], capture_output=True, text=True)
    assert r.returncode == 0, r.stdout + r.stderr
    assert (site / "ringattention_b200" / "csrc" / "attn_fwd_sm100.cu").exists()
    code = ("import ctypes, ringattention_b200.ops._lib as L; "
            f"assert str(L.LIB_PATH).startswith({str(site)!r}), L.LIB_PATH; "
            "h = ctypes.CDLL(str(L.LIB_PATH)); assert hasattr(h, 'ra_attn_fwd'); print('ok')")
    env = dict(os.environ, PYTHONPATH=str(site), RINGATTN_B200_NO_AUTOBUILD="1")
    r = subprocess.run([sys.executable, "-c", code], capture_output=True, text=True, env=env, cwd=str(tmp_path))
    assert r.returncode == 0 and "ok" in r.stdout, r.stdout + r.stderr
