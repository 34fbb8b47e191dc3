"""The Gedunex model through the engine's host side on the CPU (float32, torch stand-ins for the kernels) against the plain
implementation; configuration parsing; tensors a checkpoint may hold or not.  The GPU tests run the same cases on the real kernels."""

import json
import warnings

import numpy as np
import pytest

from dli_b200.config.gedunex import GedunexConfig, gedunex_model_spec
from dli_b200.config.llama import UnsupportedModelError
from tests import cpu_ops, gedunex_suite as suite
from tests.plain import gedunex_plain as plain


@pytest.mark.parametrize("case", suite.CASES, ids=lambda f: f.__name__[5:])
def test_case(case, tmp_path):
    with cpu_ops.patched():
        case(tmp_path, "cpu", "float32")


def test_configuration_is_checked():
    good = suite.CONFIGS["mixed"]
    parsed = GedunexConfig.from_dict(good)
    assert parsed.layers[0].mixer.window == 13 and parsed.layers[1].mixer.gate_cap == 9.0 and parsed.layers[2].mixer.softcap == 7.0
    assert parsed.layers[0].mlp.top == 2 and parsed.layers[1].mlp.kind == "dense" and parsed.embedding_scale == 3.0
    for path, value in ((("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "type"), "other"), (("layers", 0, "mlp", "kind"), "sparse"),
                        (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 1, "mixer", "gate_cap"), 0), (("layers", 0, "mixer", "softcap"), -1),
                        (("layers", 0, "mixer", "q_temp", "every"), 0), (("layers", 0, "mlp", "router", "top"), 7), (("layers", 1, "mixer", "dim"), 0),
                        (("layers", 2, "mixer", "vdim"), 17), (("layers", 0, "mixer", "scale"), 0), (("layers",), [])):
        bad = json.loads(json.dumps(good))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(UnsupportedModelError):
            GedunexConfig.from_dict(bad)
    bad = json.loads(json.dumps(good))
    del bad["layers"][1]["mixer"]["gate_cap"]
    with pytest.raises(KeyError):
        GedunexConfig.from_dict(bad)
    extra = json.loads(json.dumps(good))
    extra["layers"][1]["mixer"]["surprise"] = 1
    with warnings.catch_warnings(record=True) as seen:
        warnings.simplefilter("always")
        assert GedunexConfig.from_dict(extra) == parsed  # a key the parser does not know is reported, not obeyed
    assert any("surprise" in str(w.message) for w in seen)


def test_the_source_of_mixed_values_is_the_first_layer_that_mixes():
    spec = gedunex_model_spec(GedunexConfig.from_dict(suite.CONFIGS["memory_first"]))
    assert [layer.parts["mixer"].params.get("value_mix") for layer in spec.layers] == [None, None, "source", "mix"]


def test_a_mixing_factor_that_mixes_nothing_may_be_stored_or_not(tmp_path):
    """The source layer's own factor is not read: a checkpoint with it and one without it load and compute the same."""
    import dli_b200
    from dli_b200.weights import write_safetensors
    from tests.plain.llama_plain import read_safetensors
    import torch

    cfg = suite.CONFIGS["mixed"]
    w = suite.make_model(tmp_path / "m", cfg, seed=2)
    stored = read_safetensors(tmp_path / "m" / "model.safetensors")
    assert "l0.mix.vmix" in stored
    less = {k: torch.from_numpy(v.copy()) for k, v in stored.items() if k != "l0.mix.vmix"}
    (tmp_path / "less").mkdir()
    (tmp_path / "less" / "config.json").write_text(json.dumps(cfg))
    write_safetensors(tmp_path / "less" / "model.safetensors", less)
    toks = suite.tokens_for(cfg, 20, seed=1)
    with cpu_ops.patched():
        a, b = (suite.Session(tmp_path / d, "cpu", "float32").whole("a", toks) for d in ("m", "less"))
        assert np.array_equal(a, b)
        suite.close(a, plain.forward(cfg, w, toks), "float32")
        del less["l2.mix.vmix"]
        write_safetensors(tmp_path / "less" / "model.safetensors", less)
        with pytest.raises(ValueError, match="l2.mix.vmix"):
            dli_b200.load_model(tmp_path / "less", "float32", "cpu")
