"""How the kernel sources become libraries, on the CPU: every entry point of the C interface has a source, a model names the
sources it needs, entry points compile their own source only, and the whole library serves where it is there."""
import ctypes
import os
import re
import shutil

import pytest
import torch

import citlali_b200 as cb
from citlali_b200.csrc import build
from citlali_b200.engine.model import DecoderModel
from citlali_b200.parts.base import BuildContext
from nomutar_models import CONFIGS, config


def test_every_entry_point_has_one_source():
    owner = {}
    for f in build.sources():
        with open(os.path.join(build._HERE, f)) as fh:
            for symbol in build._ENTRY.findall(fh.read()):
                assert symbol not in owner, f"{symbol} is defined in {owner.get(symbol)} and in {f}"
                owner[symbol] = f
    declared = set()
    for h in ("api.h", "no_alloc.h"):
        with open(os.path.join(build._HERE, h)) as fh:
            code = re.sub(r"//[^\n]*", "", fh.read())
        declared |= set(re.findall(r"\b(citlali_\w+)\s*\(", code))
    assert declared <= set(owner), declared - set(owner)


def test_models_name_existing_sources():
    known = {f[:-3] for f in build.sources()}
    for name in CONFIGS:
        for dtype in (torch.float32, torch.bfloat16):
            named = DecoderModel(config(name).to_model_spec(), BuildContext(torch.device("cpu"), dtype)).kernel_sources()
            assert set(named) <= known and "elementwise" in named and "group_norm" in named
            assert not ({"delta_rule", "latent_attention", "sigmoid_attention", "hyper_connection"} & set(named))
    q = cb.config_from_dict(dict(architectures=["Qwen3ForCausalLM"], num_hidden_layers=1, hidden_size=64, num_attention_heads=2,
                                 num_key_value_heads=1, head_dim=32, intermediate_size=64, vocab_size=50, rope_theta=1e4, rms_norm_eps=1e-6,
                                 tie_word_embeddings=True, max_position_embeddings=64))
    named = DecoderModel(q.to_model_spec(), BuildContext(torch.device("cpu"), torch.float32)).kernel_sources()
    assert named == ["attention_generic", "elementwise", "gemm_simt"]


def test_an_entry_point_compiles_its_own_source_only(tmp_path, monkeypatch):
    if shutil.which("nvcc") is None and not os.path.isfile("/usr/local/cuda/bin/nvcc"):
        pytest.skip("no nvcc here")
    monkeypatch.setattr(build, "_build_dir", lambda: str(tmp_path))
    kernels = build.Kernels()
    assert kernels._whole is None and kernels._loaded == {}
    assert kernels.citlali_argmax_rows is not None
    built = lambda: sorted(f for f in os.listdir(tmp_path) if f.endswith(".o"))
    assert built() == ["elementwise.o", "sampling.o"] and set(kernels._loaded) == {"elementwise", "sampling"}
    kernels.citlali_last_error.restype = ctypes.c_char_p
    # a refusal's text crosses from one library to the other
    code = kernels.citlali_soft_cap(None, ctypes.c_size_t(4), ctypes.c_float(-1.0), None)
    assert code < 0 and b"soft_cap" in kernels.citlali_last_error()
    with pytest.raises(AttributeError):
        kernels.citlali_no_such_entry
    stamp = os.path.getmtime(tmp_path / "sampling.o")
    again = build.Kernels()                                # nothing is compiled twice
    again.prepare(["sampling"])
    assert os.path.getmtime(tmp_path / "sampling.o") == stamp
