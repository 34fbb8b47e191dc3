"""Typed configuration of the Novunex decoder, and its model as parts.

A Novunex layer reads the residual stream itself and norms only what its sublayers return: x <- x + N1(mixer(x)), then
x <- x + N2(ff(x)) (RMS norms; the feed-forward may be absent).  The mixer is grouped-query softmax attention with rotation whose
values have a size of their own, in two forms: ``attention`` norms every query and key head and adds one to the softmax's
denominator (a sink of score 0), ``attention_2`` norms the whole query and key projections and scales the rotation's
frequencies by wavelength.  A layer may read an earlier layer's keys and values.  The feed-forward is a routed mixture of
squared-relu ones (softmax over all router outputs, a correction that only steers the choice, weights as they are), the last
router outputs being the identity, with a shared feed-forward beside it.  config.json gives every size and constant, layer by
layer; nothing here is fixed to one model.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .llama import UnsupportedModelError
from .pazenex import _positive
from .spec import LayerSpec, ModelSpec, PartSpec, RunStep
from .sugonex import _keys


@dataclass(frozen=True)
class WavelengthScaling:
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class RotaryAttentionConfig:
    kind: str  # "attention" | "attention_2"
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int
    rot_scaling: WavelengthScaling | None
    kv_from: int | None  # the layer whose keys and values this one reads (None: its own)

    @property
    def cached_as(self) -> tuple:
        """What a layer that reads another's keys and values has to have in common with it."""
        return (self.heads, self.kv_heads, self.dim, self.vdim, self.rot_base, self.rot_dims, self.rot_scaling)


@dataclass(frozen=True)
class IdentityMoeConfig:
    ff: int  # of one expert
    experts: int
    identity: int  # router outputs behind the experts' whose output is the input
    top: int
    shared_ff: int | None


@dataclass(frozen=True)
class NovunexLayerConfig:
    mixer: RotaryAttentionConfig
    mlp: IdentityMoeConfig | None


KINDS = ("attention", "attention_2")


def _parse_mixer(kind: str, m: dict, where: str) -> RotaryAttentionConfig:
    _keys(m, where, ("heads", "kv_heads", "dim", "vdim", "scale"), ("rot", "kv_from"))
    heads, kv_heads, dim, vdim = (_positive(m[k], f"{where}.{k}") for k in ("heads", "kv_heads", "dim", "vdim"))
    if heads % kv_heads:
        raise UnsupportedModelError(f"{where}.heads={heads} is not a multiple of kv_heads={kv_heads}")
    scale = float(m["scale"])
    if not scale > 0:
        raise UnsupportedModelError(f"{where}.scale={scale} must be positive")
    base, dims, scaling = 10000.0, 0, None
    if m.get("rot") is not None:
        _keys(m["rot"], where + ".rot", ("base", "dims"), ("scaling",))
        base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
        if dims % 2 or not 0 <= dims <= dim or not base > 0:
            raise UnsupportedModelError(f"{where}.rot: dims={dims} must be even and at most dim={dim}, base={base} positive")
        if m["rot"].get("scaling") is not None:
            s = m["rot"]["scaling"]
            _keys(s, where + ".rot.scaling", ("factor", "low", "high", "original"))
            scaling = WavelengthScaling(float(s["factor"]), float(s["low"]), float(s["high"]), float(s["original"]))
            if not (scaling.factor > 0 and scaling.original > 0 and 0 < scaling.low < scaling.high):
                raise UnsupportedModelError(f"{where}.rot.scaling: factor and original must be positive, low positive and below high")
    kv_from = m.get("kv_from")
    return RotaryAttentionConfig(kind, heads, kv_heads, dim, vdim, scale, base, dims, scaling, None if kv_from is None else int(kv_from))


def _parse_mlp(m: dict, where: str) -> IdentityMoeConfig:
    _keys(m, where, ("kind", "expert", "router"), ("shared",))
    if m["kind"] != "moe":
        raise UnsupportedModelError(f"{where}.kind={m['kind']!r} (known: moe)")
    _keys(m["expert"], where + ".expert", ("ff",))
    _keys(m["router"], where + ".router", ("experts", "top"), ("identity",))
    experts, top = _positive(m["router"]["experts"], where + ".router.experts"), _positive(m["router"]["top"], where + ".router.top")
    identity = int(m["router"].get("identity") or 0)
    if identity < 0 or top > experts + identity:
        raise UnsupportedModelError(f"{where}.router: {experts} experts and {identity} identities cannot yield {top} choices")
    shared = None
    if m.get("shared") is not None:
        _keys(m["shared"], where + ".shared", ("ff",))
        shared = _positive(m["shared"]["ff"], where + ".shared.ff")
    return IdentityMoeConfig(_positive(m["expert"]["ff"], where + ".expert.ff"), experts, identity, top, shared)


@dataclass(frozen=True)
class NovunexConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple[NovunexLayerConfig, ...]

    @classmethod
    def from_dict(cls, cfg: dict[str, Any]) -> "NovunexConfig":
        _keys(cfg, "config", ("architecture", "layers", "norm", "vocab", "width"))
        _keys(cfg["norm"], "norm", ("eps",))
        if not isinstance(cfg["layers"], list) or not cfg["layers"]:
            raise UnsupportedModelError("layers must be a list with at least one layer")
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            where = f"layers[{i}]"
            _keys(entry, where, ("type", "mixer"), ("mlp",))
            if entry["type"] not in KINDS:
                raise UnsupportedModelError(f"{where}.type={entry['type']!r} (known: {', '.join(KINDS)})")
            m = _parse_mixer(entry["type"], entry["mixer"], where + ".mixer")
            if m.kv_from is not None:
                src = layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if src is None or src.kv_from is not None:
                    raise UnsupportedModelError(f"{where}.mixer.kv_from={m.kv_from} must name an earlier layer with keys and values of its own")
                if src.cached_as != m.cached_as:
                    raise UnsupportedModelError(f"{where}.mixer reads layer {m.kv_from}'s keys and values, but its heads, sizes or rotation differ")
            layers.append(NovunexLayerConfig(m, None if entry.get("mlp") is None else _parse_mlp(entry["mlp"], where + ".mlp")))
        return cls(_positive(cfg["vocab"], "vocab"), _positive(cfg["width"], "width"), float(cfg["norm"]["eps"]), tuple(layers))


def _position(m: RotaryAttentionConfig) -> PartSpec:
    params: dict[str, Any] = {"head_dim": m.dim, "rotary_dim": m.rot_dims, "theta": m.rot_base, "exact": True}
    if m.rot_scaling is not None:
        s = m.rot_scaling
        params.update({"scaling": "llama3", "factor": s.factor, "low_freq_factor": s.low, "high_freq_factor": s.high,
                       "original_max_position_embeddings": s.original})
    return PartSpec("rotary", params)


def novunex_model_spec(cfg: NovunexConfig) -> ModelSpec:
    """Tensor names: ``embed``, ``head``, ``final.norm``; layer i's tensors start with ``l<i>.``: ``norm1`` (behind the mixer), ``norm2``
    (behind the feed-forward), ``mix.*``, ``mlp.router``, ``mlp.correction``, ``mlp.e<j>.*``, ``mlp.shared.*``."""
    W = cfg.width

    def out_norm(name: str) -> PartSpec:
        return PartSpec("group_rmsnorm", {"size": W, "eps": cfg.eps, "tensor": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        names = {role: p + "mix." + role for role in ("q", "k", "v", "o")}
        names.update({"q_norm": p + "mix.q.norm", "k_norm": p + "mix.k.norm"})
        first = m.kind == "attention"
        mixer = PartSpec("sink_attention", {
            "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "scale": m.scale,
            "position": _position(m), "sink": 0.0 if first else None, "qk_norm_eps": cfg.eps, "qk_norm": "head" if first else "projection",
            "own_kv": m.kv_from is None, "pad_rows": True, "tensors": names}, p + "mix.")
        parts = {"mixer": mixer, "mixer_post_norm": out_norm(p + "norm1")}
        f = layer.mlp
        if f is not None:
            shared = None
            if f.shared_ff is not None:
                shared = PartSpec("dense_act", {"hidden_size": W, "intermediate_size": f.shared_ff, "activation": "relu2",
                                                "tensors": {"up": p + "mlp.shared.up", "down": p + "mlp.shared.down"}}, p + "mlp.shared.")
            parts["ffn"] = PartSpec("routed_mlp", {
                "hidden_size": W, "intermediate_size": f.ff, "num_experts": f.experts, "identity": f.identity, "top": f.top, "activation": "relu2",
                "gated": False, "score": "softmax", "shared": shared,
                "tensors": {"router": p + "mlp.router", "correction": p + "mlp.correction", "up": p + "mlp.e{}.up", "down": p + "mlp.e{}.down"}}, p + "mlp.")
            parts["ffn_post_norm"] = out_norm(p + "norm2")
        layers.append(LayerSpec("outnorm", parts))
    return ModelSpec(
        hidden_size=W,
        vocab_size=cfg.vocab,
        # (without a second table this is the plain embedding that also leaves the stream in the activation dtype, which the first product reads)
        embedding=PartSpec("pair_hash_embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "tensor": "embed"}),
        layers=tuple(layers),
        run_order=tuple(RunStep(i, cache_of=layer.mixer.kv_from) for i, layer in enumerate(cfg.layers)),
        final_norm=PartSpec("group_rmsnorm", {"size": W, "eps": cfg.eps, "tensor": "final.norm"}),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tensor": "head"}),
    )
