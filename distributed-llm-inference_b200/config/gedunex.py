"""Typed configuration of the Gedunex decoder, and its model as parts.

A Gedunex layer reads the residual stream once, behind one RMS norm, and adds both of its sublayers' outputs to it,
h = N(x), x <- x + (mixer(h) + ff(h)).  The mixer is ``mlstm`` (a matrix memory with exponential gates kept as logarithms) or
``attention`` (grouped-query softmax attention without rotation: biased projections, a norm over the whole q and k
projections, a temperature on the queries that grows with the position, soft-capped scores, a distance penalty per head, a
sliding window, a learned sink per head, and values mixed with those of the first layer that mixes).  The feed-forward is a
dense gated one, a routed mixture of small ones (softmax over the chosen experts' logits), or absent.  The embedding is
scaled, and a sinusoidal position vector is added to it.  config.json gives every size and constant; nothing here is fixed to
one model.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .llama import UnsupportedModelError
from .pazenex import _positive
from .spec import LayerSpec, ModelSpec, PartSpec, looped_run_order
from .sugonex import _keys

POSITION_BASE = 10000.0  # of the sinusoidal position vectors


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    kind = "mlstm"


@dataclass(frozen=True)
class CappedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float | None
    window: int | None
    temp_coef: float  # 0: no temperature
    temp_every: float
    v_mix: bool

    kind = "attention"


@dataclass(frozen=True)
class GedunexMlpConfig:
    kind: str  # "dense" | "moe"
    ff: int  # of the dense feed-forward, or of one expert
    experts: int = 0
    top: int = 0


@dataclass(frozen=True)
class GedunexLayerConfig:
    mixer: MatrixMemoryConfig | CappedAttentionConfig
    mlp: GedunexMlpConfig | None


def _parse_mlstm(m: dict, where: str) -> MatrixMemoryConfig:
    _keys(m, where, ("heads", "dim", "vdim", "gate_cap"))
    cap = float(m["gate_cap"])
    if not cap > 0:
        raise UnsupportedModelError(f"{where}.gate_cap={cap} must be positive")
    return MatrixMemoryConfig(*(_positive(m[k], f"{where}.{k}") for k in ("heads", "dim", "vdim")), cap)


def _parse_attention(m: dict, where: str) -> CappedAttentionConfig:
    _keys(m, where, ("heads", "kv_heads", "dim", "vdim", "scale"), ("softcap", "mask", "q_temp", "v_mix"))
    heads, kv_heads, dim, vdim = (_positive(m[k], f"{where}.{k}") for k in ("heads", "kv_heads", "dim", "vdim"))
    if heads % kv_heads:
        raise UnsupportedModelError(f"{where}.heads={heads} is not a multiple of kv_heads={kv_heads}")
    scale = float(m["scale"])
    if not scale > 0:
        raise UnsupportedModelError(f"{where}.scale={scale} must be positive")
    cap = None if m.get("softcap") is None else float(m["softcap"])
    if cap is not None and not cap > 0:
        raise UnsupportedModelError(f"{where}.softcap={cap} must be positive (or absent)")
    window = None
    if m.get("mask") is not None:
        _keys(m["mask"], where + ".mask", ("size",))
        window = _positive(m["mask"]["size"], where + ".mask.size")
    coef, every = 0.0, 1.0
    if m.get("q_temp") is not None:
        _keys(m["q_temp"], where + ".q_temp", ("coef", "every"))
        coef, every = float(m["q_temp"]["coef"]), float(m["q_temp"]["every"])
        if not every > 0:
            raise UnsupportedModelError(f"{where}.q_temp.every={every} must be positive")
    return CappedAttentionConfig(heads, kv_heads, dim, vdim, scale, cap, window, coef, every, bool(m.get("v_mix", False)))


def _parse_mlp(m: dict, where: str) -> GedunexMlpConfig:
    kind = m.get("kind") if isinstance(m, dict) else None
    if kind == "dense":
        _keys(m, where, ("kind", "ff"))
        return GedunexMlpConfig("dense", _positive(m["ff"], where + ".ff"))
    if kind == "moe":
        _keys(m, where, ("kind", "expert", "router"))
        _keys(m["expert"], where + ".expert", ("ff",))
        _keys(m["router"], where + ".router", ("experts", "top"))
        experts, top = _positive(m["router"]["experts"], where + ".router.experts"), _positive(m["router"]["top"], where + ".router.top")
        if top > experts:
            raise UnsupportedModelError(f"{where}.router: {experts} experts cannot yield {top} choices")
        return GedunexMlpConfig("moe", _positive(m["expert"]["ff"], where + ".expert.ff"), experts, top)
    raise UnsupportedModelError(f"{where}.kind={kind!r} (known: dense, moe)")


_MIXERS = {"mlstm": "_parse_mlstm", "attention": "_parse_attention"}  # looked up by name at every call


@dataclass(frozen=True)
class GedunexConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: tuple[GedunexLayerConfig, ...]

    @classmethod
    def from_dict(cls, cfg: dict[str, Any]) -> "GedunexConfig":
        _keys(cfg, "config", ("architecture", "layers", "norm", "vocab", "width"), ("embedding",))
        _keys(cfg["norm"], "norm", ("eps",))
        emb = cfg.get("embedding") or {}
        _keys(emb, "embedding", (), ("scale",))
        if not isinstance(cfg["layers"], list) or not cfg["layers"]:
            raise UnsupportedModelError("layers must be a list with at least one layer")
        layers = []
        mixing = None  # kv_heads * vdim of the layers that mix values
        for i, entry in enumerate(cfg["layers"]):
            where = f"layers[{i}]"
            _keys(entry, where, ("type", "mixer"), ("mlp",))
            if entry["type"] not in _MIXERS:
                raise UnsupportedModelError(f"{where}.type={entry['type']!r} (known: {', '.join(_MIXERS)})")
            mixer = globals()[_MIXERS[entry["type"]]](entry["mixer"], where + ".mixer")
            if isinstance(mixer, CappedAttentionConfig) and mixer.v_mix:
                size = mixer.kv_heads * mixer.vdim
                if mixing is not None and size != mixing:
                    raise UnsupportedModelError(f"{where}.mixer: {size} numbers of values a token cannot be mixed with the first mixing layer's {mixing}")
                mixing = size
            layers.append(GedunexLayerConfig(mixer, None if entry.get("mlp") is None else _parse_mlp(entry["mlp"], where + ".mlp")))
        return cls(_positive(cfg["vocab"], "vocab"), _positive(cfg["width"], "width"), float(cfg["norm"]["eps"]), float(emb.get("scale", 1.0)), tuple(layers))


def gedunex_model_spec(cfg: GedunexConfig) -> ModelSpec:
    """Tensor names: ``embed``, ``head``, ``final.norm``; layer i's tensors start with ``l<i>.``: ``norm1``, ``mix.*``, ``mlp.*``
    (``mlp.gate``, ``mlp.up``, ``mlp.down``, or ``mlp.router``, ``mlp.router.b``, ``mlp.e<j>.*``)."""
    W = cfg.width

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": W, "eps": cfg.eps, "tensor": name})

    layers = []
    first_mixing = next((i for i, layer in enumerate(cfg.layers) if isinstance(layer.mixer, CappedAttentionConfig) and layer.mixer.v_mix), None)
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        if isinstance(m, CappedAttentionConfig):
            names = {role: p + "mix." + role for role in ("q", "k", "v", "o", "sink", "vmix")}
            names.update({"q_bias": p + "mix.q.b", "k_bias": p + "mix.k.b", "v_bias": p + "mix.v.b", "q_norm": p + "mix.q.norm", "k_norm": p + "mix.k.norm"})
            value_mix = None if not m.v_mix else ("source" if i == first_mixing else "mix")
            mixer = PartSpec("capped_attention", {
                "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "scale": m.scale,
                "window": m.window, "bias": True, "qk_norm_eps": cfg.eps, "temp_coef": m.temp_coef, "temp_every": m.temp_every, "softcap": m.softcap,
                "slopes": [2.0 ** (-8.0 * (h + 1) / m.heads) for h in range(m.heads)], "head_sinks": True, "value_mix": value_mix, "tensors": names}, p + "mix.")
        else:
            names = {role: p + "mix." + role for role in ("q", "k", "v", "i", "f", "g", "norm", "o")}
            names.update({"i_bias": p + "mix.i.b", "f_bias": p + "mix.f.b"})
            mixer = PartSpec("matrix_memory", {"hidden_size": W, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "gate_cap": m.gate_cap,
                                               "eps": cfg.eps, "tensors": names}, p + "mix.")
        parts = {"mixer_norm": norm(p + "norm1"), "mixer": mixer}
        f = layer.mlp
        if f is not None and f.kind == "dense":
            parts["ffn"] = PartSpec("glu", {"hidden_size": W, "intermediate_size": f.ff, "activation": "silu",
                                            "tensors": {"gate": p + "mlp.gate", "up": p + "mlp.up", "down": p + "mlp.down"}}, p + "mlp.")
        elif f is not None:
            parts["ffn"] = PartSpec("routed_glu", {
                "hidden_size": W, "intermediate_size": f.ff, "num_experts": f.experts, "top": f.top, "activation": "silu", "score": "softmax_chosen",
                "tensors": {"router": p + "mlp.router", "correction": p + "mlp.router.b", "gate": p + "mlp.e{}.gate", "up": p + "mlp.e{}.up",
                            "down": p + "mlp.e{}.down"}}, p + "mlp.")
        layers.append(LayerSpec("parallel", parts))
    return ModelSpec(
        hidden_size=W,
        vocab_size=cfg.vocab,
        embedding=PartSpec("sinusoid_embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "tensor": "embed", "scale": cfg.embedding_scale,
                                                  "position_base": POSITION_BASE}),
        layers=tuple(layers),
        run_order=looped_run_order(len(cfg.layers), None),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tensor": "head"}),
    )
