"""The decoder: embedding, layers in run order, final norm, head — built from a ModelSpec."""

from __future__ import annotations

import torch

from ..config.spec import ModelSpec
from ..kernels import ops
from ..kernels.gemm import SKINNY_MAX_TOKENS_HEAD, linear, project
from ..weights.loader import TensorDecl
from .base import BuildEnv, Part, ResidualStream, build_part, can_fuse, normed_input, register_part, tensor_name


@register_part("embedding", "token_embedding")
class TokenEmbedding(Part):
    """h = table[token_ids], no scale (src/dli/model/llama.py:291).  params: vocab_size, hidden_size."""

    graph_capturable = True

    def __init__(self, spec, env) -> None:
        super().__init__(spec, env)
        self.vocab, self.hidden = int(spec.params["vocab_size"]), int(spec.params["hidden_size"])
        self.name = tensor_name(spec, "weight", "weight")
        self.weight: torch.Tensor | None = None

    def declare(self):
        return {self.name: TensorDecl((self.vocab, self.hidden))}

    def load(self, tensors):
        self.weight = tensors[self.name]

    def forward(self, token_ids: torch.Tensor) -> torch.Tensor:
        h = torch.empty((token_ids.numel(), self.hidden), dtype=torch.float32, device=token_ids.device)
        ops.embedding(h, self.weight, token_ids)
        return h


@register_part("embedding", "sinusoid_embedding")
class SinusoidEmbedding(Part):
    """h = table[token] * scale + s(position): a fixed vector of sines (even places) and cosines (odd places) of the token's
    position is added, the places 2i and 2i + 1 sharing the frequency position_base^(-2i / hidden_size).  The frequencies are
    made on the host in float64 and kept as a float32 and its remainder, so that the angles of far positions keep float32's
    precision.  params: vocab_size, hidden_size, tensor, scale, position_base."""

    graph_capturable = True

    def __init__(self, spec, env) -> None:
        super().__init__(spec, env)
        p = spec.params
        self.vocab, self.hidden = int(p["vocab_size"]), int(p["hidden_size"])
        self.scale, base = float(p.get("scale", 1.0)), float(p["position_base"])
        self.name = tensor_name(spec, "weight", "weight")
        freq = torch.tensor([base ** (-2.0 * i / self.hidden) for i in range((self.hidden + 1) // 2)], dtype=torch.float64)
        head = freq.to(torch.float32)
        self.freq = torch.stack([head, (freq - head.double()).to(torch.float32)]).contiguous().to(env.device)  # [2, pairs]
        self.weight: torch.Tensor | None = None

    def declare(self):
        return {self.name: TensorDecl((self.vocab, self.hidden))}

    def load(self, tensors):
        self.weight = tensors[self.name]

    def forward_step(self, batch, cache) -> ResidualStream:
        h = torch.empty((batch.token_ids.numel(), self.hidden), dtype=torch.float32, device=batch.token_ids.device)
        ops.sinusoid_embedding(h, self.weight, self.scale, self.freq, batch.token_ids, batch.positions)
        return ResidualStream(h)


@register_part("embedding", "pair_hash_embedding")
class PairHashEmbedding(Part):
    """h = table[token] * scale + pair_table[row]: beside the token's own row, a row of a second table chosen by a hash of
    the token and the one in front of it, row = (previous * mul_prev + token * mul_cur) mod buckets; a sequence's first
    token takes the table's last row (number ``buckets``).  The token in front of a step's first one is part of the
    request's state: one int32 per state slot, which the kernel reads and then leaves the step's last token in.
    Without ``pair`` it is a scaled embedding.  params: vocab_size, hidden_size, tensor, scale, pair (tensor, buckets,
    mul_prev, mul_cur; or None)."""

    graph_capturable = True

    def __init__(self, spec, env) -> None:
        super().__init__(spec, env)
        p = spec.params
        self.vocab, self.hidden = int(p["vocab_size"]), int(p["hidden_size"])
        self.scale = float(p.get("scale", 1.0))
        self.name = tensor_name(spec, "weight", "weight")
        self.pair = p.get("pair")
        if self.pair is not None:
            self.buckets, self.mul_prev, self.mul_cur = int(self.pair["buckets"]), int(self.pair["mul_prev"]), int(self.pair["mul_cur"])
            if self.buckets < 1 or self.mul_prev < 0 or self.mul_cur < 0:
                raise ValueError("pair_hash_embedding: buckets must be positive and the multipliers not negative")
        self.weight = self.pair_table = None

    def declare(self):
        out = {self.name: TensorDecl((self.vocab, self.hidden))}
        if self.pair is not None:
            out[self.pair["tensor"]] = TensorDecl((self.buckets + 1, self.hidden))
        return out

    def load(self, tensors):
        self.weight = tensors[self.name]
        if self.pair is not None:
            self.pair_table = tensors[self.pair["tensor"]]

    def cache_need(self):
        from ..cache.needs import StateNeed

        return StateNeed((1,), torch.int32) if self.pair is not None else None

    def forward_step(self, batch, cache) -> ResidualStream:
        n = batch.token_ids.numel()
        h = torch.empty((n, self.hidden), dtype=torch.float32, device=batch.token_ids.device)
        y = torch.empty((n, self.hidden), dtype=self.env.dtype, device=h.device) if self.env.dtype != torch.float32 else None
        if self.pair is None:
            ops.pair_embedding(h, self.weight, self.scale, None, 0, 0, 0, batch.token_ids, batch.positions, batch.seq_of_token, batch.q_start,
                               batch.state_slot, None, y)
        else:
            if cache is None or cache.state is None:
                raise RuntimeError("pair_hash_embedding: the step brought no state slots for the previous token")
            ops.pair_embedding(h, self.weight, self.scale, self.pair_table, self.buckets, self.mul_prev, self.mul_cur, batch.token_ids,
                               batch.positions, batch.seq_of_token, batch.q_start, batch.state_slot, cache.state, y)
        stream = ResidualStream(h)
        stream.cast = y
        return stream


@register_part("head", "lm_head")
class LMHead(Part):
    """logits = y W^T in float32, W the embedding matrix when ``tied_to`` names it
    (src/dli/model/llama.py:304-305).  A tied checkpoint that stores the head anyway is
    accepted if both are equal (src/dli/model/loader.py:75-80).  With ``scale`` the logits are multiplied by it, and
    with ``softcap`` (a positive number c) then bent into (-c, c): c * tanh(logits / c); both in float32, one kernel.
    params: vocab_size, hidden_size, tied_to, scale, softcap."""

    graph_capturable = True
    takes_scaled_rows = True

    def __init__(self, spec, env) -> None:
        super().__init__(spec, env)
        self.vocab, self.hidden = int(spec.params["vocab_size"]), int(spec.params["hidden_size"])
        self.tied_to = spec.params.get("tied_to")
        self.scale = float(spec.params.get("scale") or 1.0)
        self.softcap = float(spec.params.get("softcap") or 0.0)
        self.name = tensor_name(spec, "weight", "weight")
        self.weight: torch.Tensor | None = None

    def declare(self):
        return {self.name: TensorDecl((self.vocab, self.hidden), optional_alias_of=self.tied_to)}

    def load(self, tensors):
        self.weight = tensors[self.tied_to or self.name]

    def forward(self, y: torch.Tensor) -> torch.Tensor:
        logits = project(y, self.weight, out_dtype=torch.float32, max_tokens=SKINNY_MAX_TOKENS_HEAD)
        if self.scale != 1.0 or self.softcap:
            ops.scale_softcap(logits, self.scale, self.softcap)
        return logits


def _walk(part) -> list[Part]:
    out = [part]
    for c in part.children():
        out.extend(_walk(c))
    return out


class DecoderModel:
    """Runs the tokens of one step through the layers, in the order ``spec.run_order`` gives."""

    def __init__(self, spec: ModelSpec, dtype: torch.dtype, device: torch.device | str) -> None:
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype} is not supported (bfloat16, float32)")
        self.spec = spec
        self.env = BuildEnv(dtype, torch.device(device))
        self.embedding = build_part("embedding", spec.embedding, self.env)
        self.layers = [build_part("arrangement", layer, self.env) for layer in spec.layers]
        self.entries = [build_part("stream_entry", entry, self.env) for entry in spec.entries]
        self.final_norm = build_part("norm", spec.final_norm, self.env)
        self.head = build_part("head", spec.head, self.env)
        self.trace_layers: list | None = None  # set to a list to collect the stream after every layer run
        self._wire_deferred_products()

    def _wire_deferred_products(self) -> None:
        """A layer may leave its last product to the norm of whatever runs after it, if every
        successor it has in the run order (or the final norm and the head) can take it."""
        order = [step.layer for step in self.spec.run_order]
        ok: dict[int, bool] = {}
        for i, layer in enumerate(order):
            if i + 1 < len(order):
                first = getattr(self.layers[order[i + 1]], "first_consumer", None)
                able = first is not None and can_fuse(*first())
            else:
                able = can_fuse(self.final_norm, self.head)
            ok[layer] = ok.get(layer, True) and able
        for layer, able in ok.items():
            defer = getattr(self.layers[layer], "defer_last_product", None)
            if defer is not None:
                defer(able)

    @property
    def dtype(self) -> torch.dtype:
        return self.env.dtype

    @property
    def device(self) -> torch.device:
        return self.env.device

    def parts(self) -> list[Part]:
        out: list[Part] = []
        for top in (self.embedding, *self.entries, *self.layers, self.final_norm, self.head):
            out.extend(_walk(top))
        return out

    def declared_tensors(self) -> dict[str, TensorDecl]:
        out: dict[str, TensorDecl] = {}
        for part in self.parts():
            for name, decl in part.declare().items():
                if name in out and out[name] != decl:
                    raise ValueError(f"tensor {name!r} is declared twice with different shapes")
                out[name] = decl
        return out

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        for part in self.parts():
            part.load(tensors)

    def cache_needs(self) -> list:
        """What each run step asks of the cache manager, as its arrangement answers ``cache_need()``: None, one
        need, or several (pages and a fixed-size state side by side).  None for a step that reads another
        step's cache.  An arrangement without that method is asked through its attribute ``mixer``."""
        needs = []
        for step in self.spec.run_order:
            layer = self.layers[step.layer]
            ask = getattr(layer, "cache_need", None) or getattr(getattr(layer, "mixer", None), "cache_need", None)
            needs.append(ask() if ask is not None and step.cache_of is None else None)
        return needs

    def embedding_need(self):
        """What the embedding keeps per request between steps (StateNeeds, or None): an embedding that reads the token in
        front of a step's first one, for instance."""
        ask = getattr(self.embedding, "cache_need", None)
        return ask() if ask is not None else None

    def forward(self, batch, caches) -> torch.Tensor:
        """Logits [k, vocab] (float32) at ``batch.logit_rows``; every token's cache entries are written."""
        batch.scratch.clear()
        embed_step = getattr(self.embedding, "forward_step", None)  # an embedding that reads more of the step than its token ids
        if embed_step is not None:
            stream = embed_step(batch, getattr(caches, "embedding", None))
        else:
            stream = ResidualStream(self.embedding.forward(batch.token_ids))
        for i, step in enumerate(self.spec.run_order):
            if step.entry is not None:
                self.entries[step.entry].apply(stream, batch)
            self.layers[step.layer].forward(stream, batch, caches[i])
            if self.trace_layers is not None:  # a debugging aid: the stream after every layer run
                self.trace_layers.append(ResidualStream(stream.h.clone(), stream.take_pending()).settle())
        if batch.logit_rows.numel() == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=self.device)
        rows = None if getattr(batch, "logits_all_rows", False) else batch.logit_rows
        y = normed_input(self.final_norm, stream.h, stream.take_pending(), self.head, rows=rows)
        return self.head.forward(y)


def declared_tensors(spec: ModelSpec) -> dict[str, TensorDecl]:
    """Names, shapes and kinds of a spec's tensors, without touching a device."""
    return DecoderModel(spec, torch.float32, "meta").declared_tensors()
