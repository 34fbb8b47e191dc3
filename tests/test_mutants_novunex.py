"""Do the CPU cases of the Novunex suite notice faults?  One-line mutants of the output-norm arrangement, the attention and its
preparation, the router, the experts and the configuration, applied in memory as in tests/test_mutants.py; a few of the
suite's cases must fail for each.  No GPU."""

import dataclasses
import tempfile
from pathlib import Path

import pytest

from dli_b200.config import novunex as config_mod
from dli_b200.config import registry as registry_mod
from dli_b200.parts import rotary as rotary_mod
from dli_b200.parts.attention import SinkAttention
from dli_b200.parts.block import OutNormBlock
from dli_b200.parts.mlp import RoutedMLP
from tests import cpu_ops, novunex_suite as suite
from tests.test_mutants import mutate

DETECTORS = (suite.case_the_first_tokens, suite.case_one_more_in_the_denominator, suite.case_identities_and_the_shared_feed_forward_matter,
             suite.case_the_correction_steers_and_does_not_weigh, suite.case_a_layer_reads_another_s_keys_and_values,
             suite.case_every_configuration_whole_prompt_and_layers)


def detect():
    for case in DETECTORS:
        with tempfile.TemporaryDirectory() as tmp, cpu_ops.patched():
            case(Path(tmp), "cpu", "float32")


SPEC = (config_mod, "novunex_model_spec")
MUTANTS = {
    "the feed-forward reads the mixer's output": (OutNormBlock, "forward", "f = self.ffn.forward(stream.activation(dtype))", "f = self.ffn.forward(a)"),
    "the feed-forward's norm is the mixer's": (OutNormBlock, "forward", "else self.ffn_post_norm.add_scaled_into", "else self.mixer_post_norm.add_scaled_into"),
    "the one in the denominator is left out": (SinkAttention, "forward", "sink=self.sink)", "sink=None)"),
    "every layer has the one in the denominator": (*SPEC, '"sink": 0.0 if first else None', '"sink": 0.0'),
    "the one is e": (*SPEC, '"sink": 0.0 if first else None', '"sink": 1.0 if first else None'),
    "heads are normed as a whole": (cpu_ops, "qk_norm_rotary_store", "z = y.reshape(n, -1, head_dim) if per_head else y",
                                    "z = y.reshape(n, -1, head_dim) if per_head else y\n        w = w.repeat(y.shape[1] // w.numel())\n        z = y"),
    "projections are normed head by head": (cpu_ops, "qk_norm_rotary_store", "z = y.reshape(n, -1, head_dim) if per_head else y",
                                            "z = y.reshape(n, -1, head_dim)\n        w = w.view(-1, head_dim)"),
    "the norms are left out": (SinkAttention, "forward", "proj, self.wq_norm, self.wk_norm,", "proj, None, None,"),
    "the scale of the scores is left out": (SinkAttention, "forward", "self.nh, self.scale, self.window", "self.nh, 1.0, self.window"),
    "values have the keys' size": (SinkAttention, "forward", "value_dim=self.dv", "value_dim=self.d"),
    "a reader reads the layer in front of its source": (*SPEC, "cache_of=layer.mixer.kv_from)", "cache_of=None if layer.mixer.kv_from is None else 1)"),
    "the rotation covers the whole head": (*SPEC, '"position": _position(m)', '"position": PartSpec("rotary", {**_position(m).params, "rotary_dim": m.dim - m.dim % 2})'),
    "long wavelengths are kept": (rotary_mod, "inverse_frequencies", "torch.where(wavelen > old / low, inv / factor, inv)", "inv"),
    "the blend runs the other way": (rotary_mod, "inverse_frequencies", "(1 - smooth) * scaled / factor + smooth * scaled", "smooth * scaled / factor + (1 - smooth) * scaled"),
    "the scaling's borders change places": (config_mod, "_position", '"low_freq_factor": s.low, "high_freq_factor": s.high', '"low_freq_factor": s.high, "high_freq_factor": s.low'),
    "neighbouring dimensions turn together": (cpu_ops, "qk_norm_rotary_store", "lo, hi = qk[..., :half].clone(), qk[..., half:rotary_dim].clone()",
                                              "lo, hi = qk[..., 0:rotary_dim:2].clone(), qk[..., 1:rotary_dim:2].clone()"),
    "the correction weighs": (cpu_ops, "moe_route", "w = s.gather(1, picked)", "w = choice.gather(1, picked)"),
    "the correction does not steer": (cpu_ops, "moe_route", "choice = s + correction", "choice = s + 0.0 * correction"),
    "the weights are renormalized": (cpu_ops, "moe_route", 'weights.copy_(w * scale)', "weights.copy_(w / w.sum(-1, keepdim=True) * scale)"),
    "the router scores by the logistic function": (RoutedMLP, "forward", "self.route_scale, self.score)", 'self.route_scale, "sigmoid")'),
    "the softmax runs over the experts alone": (cpu_ops, "moe_route", "s = torch.softmax(s, -1)", "s = torch.exp(s) / torch.exp(s[:, :-1]).sum(-1, keepdim=True)"),
    "identities return nothing": (cpu_ops, "moe_experts", "weights[rows, k, None] * x[rows].float()", "weights[rows, k, None] * 0.0"),
    "identities are not weighted": (cpu_ops, "moe_experts", "weights[rows, k, None] * x[rows].float()", "x[rows].float()"),
    "the shared feed-forward is left out": (RoutedMLP, "forward", "gated=self.gated, shared=shared)", "gated=self.gated, shared=None)"),
    "relu is not squared": (cpu_ops, "moe_experts", "hidden = _plain_act(inner, activation).to(x.dtype)", "hidden = torch.relu(inner).to(x.dtype)"),
    "the activation is silu": (*SPEC, '"activation": "relu2",\n                "gated": False', '"activation": "silu",\n                "gated": False'),
    "the shared feed-forward's activation is silu": (*SPEC, '"activation": "relu2",\n                                                "tensors": {"up": p + "mlp.shared.up"',
                                                     '"activation": "silu",\n                                                "tensors": {"up": p + "mlp.shared.up"'),
}


@pytest.mark.timeout(300)
@pytest.mark.parametrize("name", list(MUTANTS), ids=lambda n: n.replace(" ", "_"))
def test_novunex_mutant_is_noticed(name, monkeypatch):
    owner, method, old, new = MUTANTS[name]
    mutate(monkeypatch, owner, method, old, new)
    if owner is cpu_ops:  # the stand-in table holds the function itself
        monkeypatch.setitem(cpu_ops.OPS, method, getattr(cpu_ops, method))
    if method == "novunex_model_spec":  # the registry holds the function itself
        monkeypatch.setitem(registry_mod._ARCHITECTURES, "Novunex",
                            dataclasses.replace(registry_mod._ARCHITECTURES["Novunex"], model_spec=config_mod.novunex_model_spec))
    with pytest.raises(Exception):  # a wrong number (AssertionError), or a folder that no longer loads
        detect()


def test_without_a_mutant_the_cases_pass():
    detect()
