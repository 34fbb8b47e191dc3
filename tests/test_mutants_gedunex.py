"""Do the CPU cases of the Gedunex suite notice faults?  One-line mutants of the one-norm parallel layer, the capped attention and
its preparation, the matrix memory, the router, the embedding and the configuration, applied in memory as in
tests/test_mutants.py; a few of the suite's cases must fail for each.  No GPU."""

import dataclasses
import tempfile
from pathlib import Path

import pytest

from dli_b200.config import gedunex as config_mod
from dli_b200.config import registry as registry_mod
from dli_b200.parts import block as block_mod
from dli_b200.parts.attention import CappedAttention
from dli_b200.parts.mlp import RoutedMLP
from dli_b200.parts.model import SinusoidEmbedding
from dli_b200.parts.ssm import MatrixMemory
from tests import cpu_ops, gedunex_suite as suite
from tests.test_mutants import mutate

DETECTORS = (suite.case_every_configuration_whole_prompt_and_layers, suite.case_the_first_tokens, suite.case_a_sink_takes_the_mass,
             suite.case_values_are_mixed_with_the_first_mixing_layer_s, suite.case_prefill_then_token_by_token)


def detect():
    for case in DETECTORS:
        with tempfile.TemporaryDirectory() as tmp, cpu_ops.patched():
            case(Path(tmp), "cpu", "float32")


MUTANTS = {
    "the feed-forward reads the mixer's output": (block_mod.ParallelBlock, "forward", "stream.pending = PendingSum(a, self.ffn.forward(y))",
                                                  "stream.pending = PendingSum(a, self.ffn.forward(a))"),
    "the feed-forward is left out": (block_mod.ParallelBlock, "forward", "stream.pending = PendingSum(a, self.ffn.forward(y))", "stream.pending = PendingSum(a, None)"),
    "the soft cap is left out": (CappedAttention, "forward", "softcap=self.softcap,", "softcap=None,"),
    "the distance costs nothing": (CappedAttention, "forward", "slopes=self.slopes)", "slopes=None)"),
    "the sinks are left out": (CappedAttention, "forward", "sink=self.sinks,", "sink=None,"),
    "the temperature is left out": (CappedAttention, "forward", "batch.positions, self.temp, source", "batch.positions, (0.0, 1.0), source"),
    "the values are mixed with none": (CappedAttention, "forward", "self.lam if mixed else None", "0.0 if mixed else None"),
    "the source's values are halved": (CappedAttention, "forward", 'elif mixed:\n        source = batch.scratch["value_source"]',
                                       'elif mixed:\n        source = batch.scratch["value_source"] * 0.5'),
    "the scale of the scores is left out": (CappedAttention, "forward", "self.nh, self.scale, self.window", "self.nh, 1.0, self.window"),
    "the padding of the output rows is forgotten": (CappedAttention, "load", "zero_padded_heads(tensors[nm[\"o\"]], self.nh, self.dv, self.row)", "tensors[nm[\"o\"]]"),
    "the biases are left out": (CappedAttention, "forward", "project_bias(x, self.w_in, self.b_in), None", "project(x, self.w_in), None"),
    "the temperature counts positions from zero": (cpu_ops, "qk_norm_mix_store", "(positions + 1).float()", "positions.float()"),
    "the slope grows towards the start": (cpu_ops, "paged_attention_simt", "slopes[:, None] * (p - keys)[None, :].float()", "slopes[:, None] * keys[None, :].float()"),
    "the two gates change places": (MatrixMemory, "load", 'torch.cat([t["i"], t["f"]], 0)', 'torch.cat([t["f"], t["i"]], 0)'),
    "the gates' biases change places": (MatrixMemory, "load", 'torch.cat([t["i_bias"], t["f_bias"]], 0)', 'torch.cat([t["f_bias"], t["i_bias"]], 0)'),
    "the memory's output is not divided": (MatrixMemory, "forward", "divisor=divisor)", "divisor=None)"),
    "the memory's gate is SiLU": (MatrixMemory, "forward", 'gate_after=True, gate="sigmoid", divisor', "gate_after=True, divisor"),
    "the memory's norm runs over all heads": (MatrixMemory, "forward", 'w["norm"], self.heads, self.eps, gate_after=True, gate="sigmoid", divisor=divisor)',
                                              'w["norm"], 1, self.eps, gate_after=True, gate="sigmoid", divisor=divisor[:, :1].contiguous())'),
    "the divisor has no floor": (cpu_ops, "matrix_memory_scan", "torch.maximum(out[:, dv].abs(), torch.exp(-m)) + 1e-6", "out[:, dv].abs() + 1e-6"),
    "the router's weights are taken over all experts": (cpu_ops, "moe_route", "torch.softmax(logits.gather(1, picked), -1) * scale",
                                                        "torch.softmax(logits, -1).gather(1, picked) * scale"),
    "the router scores by the logistic function": (RoutedMLP, "forward", "self.route_scale, self.score)", 'self.route_scale, "sigmoid")'),
    "the embedding's scale is left out": (SinusoidEmbedding, "forward_step", "self.weight, self.scale,", "self.weight, 1.0,"),
    "sines and cosines change places": (cpu_ops, "sinusoid_embedding", "torch.stack([ang.sin(), ang.cos()], -1)", "torch.stack([ang.cos(), ang.sin()], -1)"),
    "the window is read one token too wide": (config_mod, "_parse_attention", 'window = _positive(m["mask"]["size"], where + ".mask.size")',
                                              'window = _positive(m["mask"]["size"], where + ".mask.size") + 1'),
    "the slopes start at head one": (config_mod, "gedunex_model_spec", "2.0 ** (-8.0 * (h + 1) / m.heads)", "2.0 ** (-8.0 * h / m.heads)"),
    "the first layer is the source whether it mixes or not": (config_mod, "gedunex_model_spec", "and layer.mixer.v_mix), None)", "), None)"),
}


@pytest.mark.timeout(300)
@pytest.mark.parametrize("name", list(MUTANTS), ids=lambda n: n.replace(" ", "_"))
def test_gedunex_mutant_is_noticed(name, monkeypatch):
    owner, method, old, new = MUTANTS[name]
    mutate(monkeypatch, owner, method, old, new)
    if owner is cpu_ops:  # the stand-in table holds the function itself
        monkeypatch.setitem(cpu_ops.OPS, method, getattr(cpu_ops, method))
    if method == "gedunex_model_spec":  # the registry holds the function itself
        monkeypatch.setitem(registry_mod._ARCHITECTURES, "Gedunex",
                            dataclasses.replace(registry_mod._ARCHITECTURES["Gedunex"], model_spec=config_mod.gedunex_model_spec))
    with pytest.raises(Exception):  # a wrong number (AssertionError), or a folder that no longer loads
        detect()


def test_without_a_mutant_the_cases_pass():
    detect()
