"""The Novunex model through the engine's host side on the CPU (float32, torch stand-ins for the kernels) against the plain
implementation; configuration parsing; cache sharing.  The GPU tests run the same cases on the real kernels."""

import json
import warnings

import numpy as np
import pytest
import torch

from dli_b200.cache.needs import PagedKVNeed
from dli_b200.config.llama import UnsupportedModelError
from dli_b200.config.novunex import NovunexConfig, novunex_model_spec
from dli_b200.parts.model import DecoderModel
from dli_b200.parts.rotary import inverse_frequencies
from tests import cpu_ops, novunex_suite as suite
from tests.plain import novunex_plain as plain


@pytest.mark.parametrize("case", suite.CASES, ids=lambda f: f.__name__[5:])
def test_case(case, tmp_path):
    with cpu_ops.patched():
        case(tmp_path, "cpu", "float32")


def test_configuration_is_checked():
    good = suite.CONFIGS["mixed"]
    parsed = NovunexConfig.from_dict(good)
    assert parsed.layers[0].mixer.rot_scaling.original == 80 and parsed.layers[3].mixer.kv_from == 0 and parsed.layers[1].mixer.rot_scaling is None
    assert parsed.layers[0].mlp.identity == 3 and parsed.layers[0].mlp.shared_ff == 28 and parsed.layers[0].mlp.top == 3
    for path, value in ((("layers", 0, "mixer", "kv_heads"), 4), (("layers", 0, "type"), "attention_3"), (("layers", 0, "mlp", "kind"), "dense"),
                        (("layers", 0, "mixer", "rot", "dims"), 5), (("layers", 0, "mixer", "rot", "dims"), 18), (("layers", 0, "mixer", "scale"), 0),
                        (("layers", 0, "mixer", "rot", "scaling", "high"), 1.5), (("layers", 0, "mixer", "rot", "scaling", "factor"), 0),
                        (("layers", 3, "mixer", "kv_from"), 3), (("layers", 3, "mixer", "kv_from"), 1), (("layers", 3, "mixer", "vdim"), 8),
                        (("layers", 3, "mixer", "rot", "base"), 99.0), (("layers", 0, "mlp", "router", "top"), 9), (("layers", 0, "mlp", "router", "identity"), -1),
                        (("layers", 0, "mlp", "shared", "ff"), 0), (("layers",), [])):
        bad = json.loads(json.dumps(good))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(UnsupportedModelError):
            NovunexConfig.from_dict(bad)
    bad = json.loads(json.dumps(good))
    del bad["layers"][1]["mixer"]["vdim"]
    with pytest.raises(KeyError):
        NovunexConfig.from_dict(bad)
    extra = json.loads(json.dumps(good))
    extra["layers"][1]["mixer"]["surprise"] = 1
    with warnings.catch_warnings(record=True) as seen:
        warnings.simplefilter("always")
        assert NovunexConfig.from_dict(extra) == parsed  # a key the parser does not know is reported, not obeyed
    assert any("surprise" in str(w.message) for w in seen)
    chain = json.loads(json.dumps(good))
    chain["layers"].append(json.loads(json.dumps(chain["layers"][3])))
    chain["layers"][4]["mixer"]["kv_from"] = 3  # a layer that itself reads another's
    with pytest.raises(UnsupportedModelError):
        NovunexConfig.from_dict(chain)


def test_layers_that_read_another_s_cache_declare_no_keys_and_values():
    cfg = suite.CONFIGS["read_by_many"]
    spec = novunex_model_spec(NovunexConfig.from_dict(cfg))
    assert [step.cache_of for step in spec.run_order] == [None, None, None, 1, 2, 2]
    model = DecoderModel(spec, torch.bfloat16, "meta")
    names = model.declared_tensors()
    for i in (3, 4, 5):
        assert not any(n.startswith((f"l{i}.mix.k", f"l{i}.mix.v")) for n in names) and f"l{i}.mix.q.norm" in names
    # rows are padded to multiples of 16 in bfloat16, keys and values each; a layer with another's cache asks for nothing
    assert model.cache_needs() == [PagedKVNeed(1, 32, value_dim=16), PagedKVNeed(4, 16), PagedKVNeed(2, 32, value_dim=48), None, None, None]
    assert DecoderModel(spec, torch.float32, "meta").cache_needs()[:3] == [PagedKVNeed(1, 32, value_dim=16), PagedKVNeed(4, 8), PagedKVNeed(2, 20, value_dim=36)]


@pytest.mark.parametrize("scaling", [None, (6.0, 1.5, 5.0, 80), (8.0, 1.0, 4.0, 4096)])
def test_frequencies_are_rounded_once(scaling):
    rot = {"base": 7000.0, "dims": 48}
    params = {"rotary_dim": 48, "theta": 7000.0, "exact": True}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
        params.update(dict(zip(("factor", "low_freq_factor", "high_freq_factor", "original_max_position_embeddings"), scaling)), scaling="llama3")
    got = inverse_frequencies(params)
    assert got.dtype == torch.float32
    assert np.abs(got.double().numpy() / plain.frequencies(rot) - 1).max() < 6.1e-8
