"""Cases that compare the engine's Novunex model with the plain implementation (tests/plain/novunex_plain.py).

Each case takes (tmp_path, device, dtype) and builds its own small configuration and weights.  The CPU tests run them on
torch stand-ins for the kernels (float32), the GPU tests on the real kernels in both dtypes.  Weights are drawn so that
faults show: sharp attention (one missing key changes the logits), scores of both signs (the one in the denominator matters),
routers that differ from token to token, corrections as large as the scores they steer.
"""

from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch

import dli_b200
from dli_b200.config.registry import resolve_architecture
from dli_b200.engine import ModelRunner
from dli_b200.parts.model import declared_tensors
from dli_b200.weights import write_safetensors
from tests.pazenex_suite import TOL, Session, close
from tests.plain import novunex_plain as plain


def first(heads=4, kv_heads=2, dim=16, vdim=8, scale=0.3, base=1000.0, rot=8):
    """A layer whose heads are normed one by one and whose softmax has one more in the denominator."""
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}}}


def second(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.35, base=10000.0, rot=16, scaling=(6.0, 1.5, 5.0, 80), kv_from=None):
    """A layer whose projections are normed as a whole and whose frequencies are scaled."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention_2", "mixer": m}


def moe(ff=20, experts=5, identity=3, top=3, shared=28):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(layers, mlps=(), width=48, vocab=89, eps=1e-5):
    """``mlps``: the layers' feed-forwards, used in turn (None: the layer has none)."""
    mlps = list(mlps) or [moe()]
    out = {"architecture": "Novunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": []}
    for i, layer in enumerate(layers):
        out["layers"].append({**layer, "mlp": mlps[i % len(mlps)]})
    return out


# sizes that differ from one another in every respect: head counts that are and are not powers of two, several heads per
# key/value head and one, values shorter and longer than keys, rows that are and are not multiples of 8 and 16, full, partial and
# no rotation, scaled frequencies or not, keys and values read by one layer, by several, by none; one choice of experts, several,
# all; with and without identities and a shared feed-forward; layers without a feed-forward
CONFIGS = {
    "mixed": config([second(), first(), first(heads=3, kv_heads=3, dim=24, vdim=40, scale=0.2, rot=24), second(kv_from=0, scale=0.5)]),
    "read_by_many": config([first(heads=6, kv_heads=1, dim=32, vdim=16, rot=4), second(heads=4, kv_heads=4, dim=8, vdim=8, rot=8, scaling=(3.0, 1.0, 2.0, 40)),
                            second(heads=8, kv_heads=2, dim=20, vdim=36, scale=0.15, rot=12), second(heads=4, kv_heads=4, dim=8, vdim=8, rot=8, scaling=(3.0, 1.0, 2.0, 40), kv_from=1),
                            second(heads=8, kv_heads=2, dim=20, vdim=36, scale=0.4, rot=12, kv_from=2), second(heads=8, kv_heads=2, dim=20, vdim=36, scale=0.25, rot=12, kv_from=2)],
                           mlps=(moe(ff=16, experts=4, identity=1, top=1, shared=40), None, moe(ff=32, experts=6, identity=0, top=6, shared=0)), width=40, eps=1e-3),
    "only_first": config([first(), first(heads=2, kv_heads=1, dim=40, vdim=72, scale=0.12, rot=16), first(heads=12, kv_heads=4, dim=8, vdim=8, rot=0)],
                         mlps=(moe(ff=64, experts=10, identity=6, top=7, shared=16), None), width=64, vocab=130),
    "only_second": config([second(scaling=None), second(heads=5, kv_heads=1, dim=48, vdim=16, scale=0.1, rot=32, base=500.0), second(heads=2, kv_heads=2, dim=16, vdim=16, rot=2)],
                          mlps=(moe(ff=24, experts=1, identity=1, top=1), moe(ff=8, experts=3, identity=0, top=2, shared=0)), vocab=61),
    # nothing a multiple of 4 or 8
    "odd_sizes": config([second(heads=3, kv_heads=3, dim=7, vdim=5, rot=6, scaling=(2.5, 1.1, 3.3, 33)), first(heads=9, kv_heads=3, dim=5, vdim=9, rot=2),
                         second(heads=3, kv_heads=3, dim=7, vdim=5, rot=6, scaling=(2.5, 1.1, 3.3, 33), kv_from=0, scale=0.9)],
                        mlps=(moe(ff=11, experts=7, identity=2, top=3, shared=13),), width=51, vocab=67),
}


def make_model(path: Path, cfg: dict, seed: int = 0, edit=None) -> dict:
    """Writes the folder; returns the tensors as float64 arrays (as stored: values a bfloat16 engine reads unchanged).
    ``edit(tensors)`` may change the tensors before they are written."""
    arch = resolve_architecture(cfg)
    decls = declared_tensors(arch.model_spec(arch.parse_config(cfg)))
    g = torch.Generator().manual_seed(seed)

    def normal(shape, std):
        return torch.randn(shape, generator=g) * std

    tensors = {}
    for name, decl in sorted(decls.items()):
        shape = tuple(decl.shape)
        if name.endswith("correction"):
            t = normal(shape, 0.15)
        elif name.endswith("q.norm") or name.endswith("k.norm"):
            t = 1.3 + normal(shape, 0.3)
        elif len(shape) == 1:
            t = 1.0 + normal(shape, 0.2)
        elif name == "embed":
            t = normal(shape, 1.0)
        elif name.endswith("router"):
            t = normal(shape, 1.2 / shape[1] ** 0.5)
        else:
            t = normal(shape, 1.0 / shape[1] ** 0.5)
        tensors[name] = t.to(torch.bfloat16).float()
    if edit is not None:
        edit(tensors)
        tensors = {k: v.to(torch.bfloat16).float() for k, v in tensors.items()}
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(path / "model.safetensors", tensors)
    return {k: v.double().numpy() for k, v in tensors.items()}


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def rounding_error(path, device, dtype, toks, want):
    """What rounding alone does to this sequence in bfloat16: the error of the whole prompt, alone, in a fresh engine."""
    if dtype == "float32":
        return 0.0
    return float(np.abs(Session(path, device, dtype, pages=len(toks) // 8 + 2).whole("alone", toks) - want).max())


def steady(cfg, dtype):
    """``cfg`` as a case runs it in ``dtype``: as it is in float32; in bfloat16 with every expert chosen.  (A token whose choice
    between two experts is a close call may take the other one than the float64 model, and over hundreds of (token, layer) pairs
    some call is always close.  Choices are compared exactly in float32, and kernel by kernel on equal inputs.)"""
    if dtype != "bfloat16":
        return cfg
    out = json.loads(json.dumps(cfg))
    for layer in out["layers"]:
        if layer.get("mlp"):
            r = layer["mlp"]["router"]
            r["top"] = r["experts"] + r.get("identity", 0)
    return out


def pick(name, dtype):
    return steady(CONFIGS[name], dtype)


# ----------------------------------------------------------------------------- cases


def case_every_configuration_whole_prompt_and_layers(tmp_path, device, dtype):
    """Whole prompts in every configuration: logits, and the stream after every layer (in float32)."""
    for name, cfg in CONFIGS.items():
        cfg = steady(cfg, dtype)
        w = make_model(tmp_path / name, cfg, seed=3)
        toks = tokens_for(cfg, 150, seed=1)
        trace = []
        want = plain.forward(cfg, w, toks, trace)
        s = Session(tmp_path / name, device, dtype)
        s.model.trace_layers = []
        close(s.whole("a", toks), want, dtype, name)
        assert len(s.model.trace_layers) == len(trace) == len(cfg["layers"]), name
        if dtype == "float32":
            for i, h in enumerate(s.model.trace_layers):
                close(h.double().cpu().numpy(), trace[i], dtype, f"{name}: stream after layer {i}")
        s.model.trace_layers = None


def case_each_mechanism_alone(tmp_path, device, dtype):
    """One layer: each mixer with nothing beside it, with its options one by one; rows that fill the slabs of the TMA-fed and tcgen05
    attention kernels and rows that leave part of one empty, keys in one and values in two and the other way round, rows that only
    the other kernels take; feed-forwards beside the simplest mixer."""
    layers = {
        "head_norm": first(rot=0),
        "head_norm_rotated": first(rot=16),
        "rotated_in_part": first(heads=2, kv_heads=2, dim=32, rot=6),
        "projection_norm": second(rot=0, scaling=None),
        "projection_norm_rotated": second(scaling=None),
        "scaled": second(scaling=(8.0, 1.0, 4.0, 64)),
        "scaled_hard": second(scaling=(30.0, 1.0, 1.5, 25), base=100.0),
        "keys_64_values_64": first(heads=5, kv_heads=1, dim=64, vdim=64, scale=0.08, rot=32),
        "keys_64_values_128": second(heads=4, kv_heads=2, dim=64, vdim=128, scale=0.1, rot=64),
        "keys_128_values_64": first(heads=4, kv_heads=2, dim=128, vdim=64, scale=0.05, rot=64),
        "keys_128_values_128": second(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.06, rot=128),
        "keys_72_values_40": first(heads=6, kv_heads=2, dim=72, vdim=40, scale=0.08, rot=48),
        "keys_40_values_104": second(heads=3, kv_heads=3, dim=40, vdim=104, scale=0.12, rot=32),
        "keys_112_values_88": second(heads=20, kv_heads=1, dim=112, vdim=88, scale=0.06, rot=16),
        "keys_160_values_48": first(heads=2, kv_heads=1, dim=160, vdim=48, scale=0.05, rot=32),
        "keys_24_values_144": first(heads=2, kv_heads=1, dim=24, vdim=144, scale=0.2, rot=24),
        "many_heads_on_one": first(heads=34, kv_heads=1, dim=16, vdim=16),
    }
    for name, layer in layers.items():
        cfg = config([layer], mlps=(None,))
        w = make_model(tmp_path / name, cfg, seed=5)
        toks = tokens_for(cfg, 90, seed=2)
        want = plain.forward(cfg, w, toks)
        s = Session(tmp_path / name, device, dtype, pages=12)
        close(s.whole("a", toks), want, dtype, name)
        s.free("a")
        got = [s.step(("b", toks[:80], list(range(80))))] + [s.step(("b", [t], [0])) for t in toks[80:]]
        close(np.concatenate(got), want, dtype, name + ", the last ten decoded")
    for name, mlp in {"one_choice": moe(ff=24, experts=4, identity=2, top=1), "three": moe(ff=16, experts=7, identity=2, top=3), "all_chosen": moe(ff=8, experts=4, identity=2, top=6),
                      "many": moe(ff=32, experts=26, identity=6, top=12, shared=64), "one_expert": moe(ff=24, experts=1, identity=0, top=1), "no_shared": moe(shared=0),
                      "more_identities": moe(ff=16, experts=2, identity=9, top=4), "wide_experts": moe(ff=136, experts=3, identity=1, top=2, shared=72),
                      "odd": moe(ff=21, experts=5, identity=2, top=2, shared=19)}.items():
        cfg = steady(config([first(heads=1, kv_heads=1, dim=8, vdim=8)], mlps=(mlp,)), dtype)
        w = make_model(tmp_path / name, cfg, seed=6)
        for n in (1, 3, 30):
            toks = tokens_for(cfg, n, seed=3)
            s = Session(tmp_path / name, device, dtype)
            close(s.whole("a", toks), plain.forward(cfg, w, toks), dtype, f"{name}, {n} tokens")


def case_the_correction_steers_and_does_not_weigh(tmp_path, device, dtype):
    """A correction that lifts an identity and two experts above all others makes every token choose them in that order, with the
    weights their own scores give."""
    cfg = config([first(heads=1, kv_heads=1, dim=8, vdim=8)], mlps=(moe(ff=16, experts=5, identity=2, top=3, shared=0),))

    def lift(t):
        t["l0.mlp.correction"] = torch.tensor([0.0, -3.0, 1.5, 3.0, 0.0, 0.0, 5.0])

    w = make_model(tmp_path / "r", cfg, seed=8, edit=lift)
    ids, weights = plain.route(np.random.default_rng(0).normal(size=(50, 48)), w, "l0.mlp.", 3)
    assert (ids == [6, 3, 2]).all() and weights.sum(1).max() < 1 and weights[:, 0].min() < 0.1
    toks = tokens_for(cfg, 25, seed=4)
    close(Session(tmp_path / "r", device, dtype).whole("a", toks), plain.forward(cfg, w, toks), dtype, "routing")


def case_identities_and_the_shared_feed_forward_matter(tmp_path, device, dtype):
    """A router that likes the identities (the stream's own direction decides), beside small experts: left out, the logits move by far
    more than the tolerance; so do they without the shared feed-forward.  Steps of one token, of a few and of many (other kernels)."""
    cfg = config([first(heads=1, kv_heads=1, dim=8, vdim=8)], mlps=(moe(ff=16, experts=3, identity=3, top=4, shared=24),))

    def like(t):
        t["l0.mlp.router"][3:] *= 2.0
        t["l0.mlp.correction"] = torch.tensor([0.0, 0.0, 0.0, 0.3, 0.3, 0.3])

    cfg = steady(cfg, dtype)
    w = make_model(tmp_path / "i", cfg, seed=9, edit=like)
    toks = tokens_for(cfg, 45, seed=4)
    want = plain.forward(cfg, w, toks)
    less = json.loads(json.dumps(cfg))
    less["layers"][0]["mlp"]["shared"] = None
    assert np.abs(plain.forward(less, w, toks) - want).max() > 0.5
    away = {**w, "l0.mlp.correction": w["l0.mlp.correction"] - np.array([0, 0, 0, 5.0, 5.0, 5.0])}
    less["layers"][0]["mlp"] = {**cfg["layers"][0]["mlp"], "router": {**cfg["layers"][0]["mlp"]["router"], "top": 3}}
    assert np.abs(plain.forward(less, away, toks) - want).max() > 0.3  # only experts are chosen
    s = Session(tmp_path / "i", device, dtype)
    got = [s.step(("a", toks[:30], list(range(30)))), s.step(("a", toks[30:32], [0, 1])), s.step(("a", toks[32:41], list(range(9))))]
    got += [s.step(("a", [t], [0])) for t in toks[41:]]
    close(np.concatenate(got), want, dtype, "identities and shared")


def case_one_more_in_the_denominator(tmp_path, device, dtype):
    """Heads whose keys all score far below zero beside heads whose keys score far above: the first ones' outputs all but vanish beside the
    others'; without the one, their weights would be ordinary ones, and the logits move by far more than the tolerance.  In a
    prompt, in portions, decoded."""
    for rows in ((16, 24), (64, 128)):
        cfg = config([first(heads=4, kv_heads=4, dim=rows[0], vdim=rows[1], scale=1.5 / rows[0] ** 0.5, rot=4)], mlps=(None,), width=32, vocab=40)

        def opposed(t):
            d = rows[0]
            mark = torch.zeros(32)
            mark[0] = 1.0
            t["embed"][:, 0] = 3.0
            for role, sign in (("q", torch.tensor([1.0, 1.0, 1.0, 1.0])), ("k", torch.tensor([-1.0, 1.0, -0.5, 0.3]))):
                rowsw = t[f"l0.mix.{role}"].view(4, d, 32)
                rowsw[:, :, 0] = sign[:, None] * torch.linspace(0.5, 1.5, d)

        w = make_model(tmp_path / f"one{rows[0]}", cfg, seed=29, edit=opposed)
        toks = tokens_for(cfg, 40, seed=8)
        want = plain.forward(cfg, w, toks)
        ordinary = {**cfg, "layers": [{**cfg["layers"][0]}]}
        ones = plain.softmax_weights
        try:
            plain.softmax_weights = lambda s, one_more: ones(s, False)
            without = plain.forward(ordinary, w, toks)
        finally:
            plain.softmax_weights = ones
        assert np.abs(without - want).max() > 0.5
        s = Session(tmp_path / f"one{rows[0]}", device, dtype)
        got = [s.step(("a", toks[:21], list(range(21)))), s.step(("a", toks[21:30], list(range(9))))] + [s.step(("a", [t], [0])) for t in toks[30:]]
        close(np.concatenate(got), want, dtype, "one more in the denominator")


def case_a_layer_reads_another_s_keys_and_values(tmp_path, device, dtype):
    """Two layers between the source and its readers, one of which would itself be a source of the right shape: reading that one's keys, or
    the reader's own stream, moves the logits by far more than the tolerance.  Prompt, portions, single tokens, requests side by side."""
    common = dict(heads=4, kv_heads=2, dim=16, vdim=24)
    cfg = config([second(**common), second(**common, scale=0.5), first(), second(**common, kv_from=0), second(**common, kv_from=1, scale=0.6), second(**common, kv_from=0, scale=0.2)],
                 mlps=(None, moe(top=8)))
    w = make_model(tmp_path / "s", cfg, seed=12)
    seqs = {"a": tokens_for(cfg, 60, seed=9), "b": tokens_for(cfg, 38, seed=10)}
    want = {r: plain.forward(cfg, w, t) for r, t in seqs.items()}
    other = json.loads(json.dumps(cfg))
    other["layers"][3]["mixer"]["kv_from"] = 1
    assert np.abs(plain.forward(other, w, seqs["a"]) - want["a"]).max() > 0.5
    s = Session(tmp_path / "s", device, dtype, pages=20, page_size=8)
    got = {r: [] for r in seqs}
    at = {r: 0 for r in seqs}
    for plan in [{"a": 25}, {"a": 3, "b": 20}, {"a": 1, "b": 1}, {"a": 1}, {"a": 17, "b": 1}, {"a": 1, "b": 13}, {"a": 10, "b": 1}, {"a": 1, "b": 1}, {"a": 1, "b": 1}]:
        parts = [(r, seqs[r][at[r] : at[r] + n], list(range(n))) for r, n in plan.items()]
        out = s.step(*parts)
        row = 0
        for r, t, _ in parts:
            got[r].append(out[row : row + len(t)])
            row += len(t)
            at[r] += len(t)
    for r in seqs:
        close(np.concatenate(got[r]), want[r][: at[r]], dtype, f"request {r}", rounding_error(tmp_path / "s", device, dtype, seqs[r], want[r]))


def case_prefill_then_token_by_token(tmp_path, device, dtype):
    """A prompt in one step, then 60 tokens one at a time, against the whole sequence at once; and a sequence fed token by token from its
    very first token."""
    for name in ("mixed", "read_by_many"):
        cfg = pick(name, dtype)
        w = make_model(tmp_path / name, cfg, seed=7)
        toks = tokens_for(cfg, 95, seed=3)
        want = plain.forward(cfg, w, toks)
        s = Session(tmp_path / name, device, dtype, pages=40)
        got = [s.step(("a", toks[:35], list(range(35))))]
        got += [s.step(("a", [t], [0])) for t in toks[35:]]
        close(np.concatenate(got), want, dtype, "prompt then decode", rounding_error(tmp_path / name, device, dtype, toks, want))
        s.free("a")
        got = [s.step(("b", [t], [0])) for t in toks[:20]]
        close(np.concatenate(got), want[:20], dtype, "token by token from the start")


def case_long_decoding(tmp_path, device, dtype):
    """A short prompt and 300 decoded tokens."""
    cfg = steady(config([second(heads=2, kv_heads=1, dim=16, vdim=8), first(heads=2, kv_heads=1, dim=16, vdim=32), second(heads=2, kv_heads=1, dim=16, vdim=8, kv_from=0)],
                        mlps=(moe(ff=16, experts=4, identity=2, top=2),), width=32), dtype)
    w = make_model(tmp_path / "l", cfg, seed=9)
    toks = tokens_for(cfg, 310, seed=4)
    want = plain.forward(cfg, w, toks)
    s = Session(tmp_path / "l", device, dtype, pages=44, page_size=8)
    s.step(("a", toks[:10], []))
    got = np.concatenate([s.step(("a", [t], [0])) for t in toks[10:]])
    close(got, want[10:], dtype, "long decoding", rounding_error(tmp_path / "l", device, dtype, toks, want))


def case_portions_of_many_sizes(tmp_path, device, dtype):
    """Portions down to two tokens and single tokens between them, cut inside pages and tiles of keys, and portions longer than a tile."""
    for name in ("mixed", "read_by_many", "only_first", "odd_sizes"):
        cfg = pick(name, dtype)
        w = make_model(tmp_path / name, cfg, seed=11)
        sizes = (2, 1, 2, 3, 1, 1, 9, 2, 16, 1, 7, 2, 17, 64, 65, 2, 33, 1, 81)
        toks = tokens_for(cfg, sum(sizes), seed=5)
        want = plain.forward(cfg, w, toks)
        s = Session(tmp_path / name, device, dtype, pages=44)
        got, at = [], 0
        for n in sizes:
            got.append(s.step(("a", toks[at : at + n], list(range(n)))))
            at += n
        close(np.concatenate(got), want, dtype, name, rounding_error(tmp_path / name, device, dtype, toks, want))


def case_batches_of_unequal_requests(tmp_path, device, dtype):
    """Up to four live requests: portions of some beside single tokens of others; a request sits out a step; the logits of each equal
    those of the request alone."""
    cfg = pick("mixed", dtype)
    w = make_model(tmp_path / "m", cfg, seed=13)
    seqs = {r: tokens_for(cfg, n, seed=20 + i) for i, (r, n) in enumerate((("a", 130), ("b", 33), ("c", 9), ("d", 41)))}
    want = {r: plain.forward(cfg, w, t) for r, t in seqs.items()}
    s = Session(tmp_path / "m", device, dtype, pages=40)
    at = {r: 0 for r in seqs}
    got = {r: [] for r in seqs}
    plan = [{"a": 17, "b": 2}, {"a": 1, "b": 20, "c": 3}, {"a": 1, "c": 1, "d": 30}, {"b": 1, "c": 1, "d": 1, "a": 9}, {"a": 2, "b": 2, "c": 2, "d": 2},
            {"a": 1, "b": 1, "c": 1, "d": 1}, {"d": 1, "c": 1}, {"a": 99, "b": 7, "d": 6}]
    for step in plan:
        parts = []
        for r, n in step.items():
            n = min(n, len(seqs[r]) - at[r])
            parts.append((r, seqs[r][at[r] : at[r] + n], list(range(n))))
        out = s.step(*parts)
        row = 0
        for r, t, _ in parts:
            got[r].append(out[row : row + len(t)])
            row += len(t)
            at[r] += len(t)
    for r in seqs:
        close(np.concatenate(got[r]), want[r][: at[r]], dtype, f"request {r}", rounding_error(tmp_path / "m", device, dtype, seqs[r], want[r]))


def case_pages_used_again(tmp_path, device, dtype):
    """A pool for two short requests: request after request takes the pages a finished one gave back, and computes what it would
    compute in a fresh engine."""
    cfg = pick("mixed", dtype)
    w = make_model(tmp_path / "m", cfg, seed=17)
    s = Session(tmp_path / "m", device, dtype, pages=8, page_size=8, max_requests=2)
    live = []
    for i, n in enumerate((30, 25, 31, 12, 28)):
        toks = tokens_for(cfg, n, seed=40 + i)
        if len(live) == 2:
            s.free(live.pop(0))
        cut = n // 2
        a = s.step((i, toks[:cut], list(range(cut))))
        b = s.step((i, toks[cut:], list(range(n - cut))))
        want = plain.forward(cfg, w, toks)
        close(np.concatenate([a, b]), want, dtype, f"request {i}", rounding_error(tmp_path / "m", device, dtype, toks, want))
        live.append(i)
    s.manager.check_invariants()


def _still(m):
    """Norm weights that take the rotated dimensions out of the scores, which then depend on the two tokens alone."""

    def edit(t):
        t["l0.mix.q.norm"].view(-1, m["dim"])[:, : m["rot"]["dims"]] = 0.0

    return edit


def _pair(cfg, w):
    """In a model of one attention layer that reads the embedding itself, whose rotated dimensions do not count, a score depends on the
    two tokens alone.  Returns a token whose last head scores one other token's key far above every other's, that token, and tokens
    whose keys it scores far below."""
    layer = cfg["layers"][0]
    m, per_head = layer["mixer"], layer["type"] == "attention"
    q = plain.normed_heads(w["embed"] @ w["l0.mix.q"].T, m["heads"], w["l0.mix.q.norm"], cfg["norm"]["eps"], per_head)[:, -1]
    k = plain.normed_heads(w["embed"] @ w["l0.mix.k"].T, m["kv_heads"], w["l0.mix.k.norm"], cfg["norm"]["eps"], per_head)[:, -1]
    s = q @ k.T * m["scale"]
    V = cfg["vocab"]
    gap = np.sort(s, 1)[:, -1] - np.median(s, 1)
    asker = int(max((t for t in range(V) if s[t].argmax() != t), key=lambda t: gap[t]))
    key = int(s[asker].argmax())
    noise = [t for t in range(V) if s[asker, t] < s[asker, key] - 10 and t != asker]
    assert len(noise) > 15
    return asker, key, noise


def case_one_far_key_decides(tmp_path, device, dtype):
    """Sequences made so that the last token's last head puts nearly all its mass on ONE key among hundreds — at a page border,
    beside one, at the very start, at the border of a tile of 128 keys: a kernel that skips or misplaces that key changes the logits by
    far more than the tolerance.  In a prompt, in a last portion of two tokens and decoded; in both kinds of layer, with rows for
    every attention kernel."""
    shapes = (first(heads=2, kv_heads=1, dim=16, vdim=24, scale=4.0, rot=4), second(heads=2, kv_heads=1, dim=16, vdim=16, scale=4.0, rot=4),
              first(heads=2, kv_heads=1, dim=72, vdim=40, scale=2.0, rot=16), second(heads=2, kv_heads=1, dim=40, vdim=104, scale=2.0, rot=8),
              second(heads=2, kv_heads=1, dim=64, vdim=64, scale=2.0, rot=16))
    for i, layer in enumerate(shapes):
        m = layer["mixer"]
        cfg = config([layer], mlps=(None,), width=32, vocab=50)
        w = make_model(tmp_path / f"far{i}", cfg, seed=19, edit=_still(m))
        asker, key, noise = _pair(cfg, w)
        s = Session(tmp_path / f"far{i}", device, dtype, pages=48, page_size=8)
        for far in (8, 15, 16, 1, 0, 127, 128, 263) if device != "cpu" or i == 0 else (15, 0, 128):
            toks = [noise[j] for j in np.random.default_rng(far).integers(0, len(noise), 330)]
            toks[far], toks[-1] = key, asker
            want = plain.forward(cfg, w, toks)
            without = list(toks)
            without[far] = noise[0]
            assert np.abs(plain.forward(cfg, w, without)[-1] - want[-1]).max() > 0.5, "the far key does not matter enough for this test"
            close(s.whole("p", toks)[-1], want[-1], dtype, f"rows {m['dim']}/{m['vdim']}: far key {far} in a prompt")
            s.free("p")
            s.step(("d", toks[:-1], []))
            close(s.step(("d", toks[-1:], [0]))[0], want[-1], dtype, f"rows {m['dim']}/{m['vdim']}: far key {far} decoded")
            s.free("d")
            s.step(("c", toks[:-2], []))
            close(s.step(("c", toks[-2:], [1]))[0], want[-1], dtype, f"rows {m['dim']}/{m['vdim']}: far key {far} in a last portion of two")
            s.free("c")


def case_far_positions_turn_by_their_own_angles(tmp_path, device, dtype):
    """Scores that hang on the distance alone (every token has nearly the same query and key, but values of its own): slow frequencies, kept, stretched and
    blended ones, over a thousand positions; in a prompt, in portions, decoded."""
    for i, layer in enumerate((second(heads=2, kv_heads=2, dim=16, vdim=16, scale=0.4, rot=16, base=3000.0, scaling=(5.0, 1.0, 4.0, 256)),
                               first(heads=2, kv_heads=1, dim=32, vdim=16, scale=0.2, rot=20, base=700.0))):
        cfg = config([layer], mlps=(None,), width=32, vocab=50)

        def alike(t):
            t["embed"][:, :8] = torch.linspace(-2.0, 2.0, 8)
            t["l0.mix.q"][:, 8:] *= 0.1
            t["l0.mix.k"][:, 8:] *= 0.1
            t["l0.mix.v"][:, :8] = 0.0

        w = make_model(tmp_path / f"turn{i}", cfg, seed=23, edit=alike)
        toks = tokens_for(cfg, 1030, seed=14)
        want = plain.forward(cfg, w, toks)
        if layer["type"] == "attention_2":
            flat = json.loads(json.dumps(cfg))
            del flat["layers"][0]["mixer"]["rot"]["scaling"]
            assert np.abs(plain.forward(flat, w, toks) - want).max() > 0.3
        s = Session(tmp_path / f"turn{i}", device, dtype, pages=70, page_size=16)
        got = [s.step(("a", toks[:600], list(range(600)))), s.step(("a", toks[600:603], [0, 1, 2])), s.step(("a", toks[603:1020], list(range(417))))]
        got += [s.step(("a", [t], [0])) for t in toks[1020:]]
        close(np.concatenate(got), want, dtype, "far positions", rounding_error(tmp_path / f"turn{i}", device, dtype, toks, want))


def case_the_first_tokens(tmp_path, device, dtype):
    """Sequences of one, two and three tokens, and a first step of one token followed by portions."""
    cfg = pick("mixed", dtype)
    w = make_model(tmp_path / "m", cfg, seed=27)
    s = Session(tmp_path / "m", device, dtype)
    for n in (1, 2, 3):
        toks = tokens_for(cfg, n, seed=70 + n)
        close(s.whole("a", toks), plain.forward(cfg, w, toks), dtype, f"{n} tokens")
        s.free("a")
    toks = tokens_for(cfg, 32, seed=75)
    got = np.concatenate([s.step(("b", toks[:1], [0])), s.step(("b", toks[1:3], [0, 1])), s.step(("b", toks[3:], list(range(29))))])
    close(got, plain.forward(cfg, w, toks), dtype, "one token, then portions")


def case_layer_sizes_of_a_larger_model(tmp_path, device, dtype):
    """Rows of 128 and 64 numbers, a prompt of 600 tokens in two portions (several tiles of queries and keys, many tokens per expert, the
    products for many tokens), then decoding."""
    cfg = config([second(heads=8, kv_heads=2, dim=128, vdim=64, scale=0.05, rot=128, scaling=(8.0, 1.0, 4.0, 400)),
                  first(heads=16, kv_heads=4, dim=64, vdim=128, scale=0.08, rot=32), second(heads=8, kv_heads=2, dim=128, vdim=64, scale=0.07, rot=128, scaling=(8.0, 1.0, 4.0, 400), kv_from=0)],
                 mlps=(moe(ff=128, experts=8, identity=4, top=3, shared=512),), width=512, vocab=300)
    cfg = steady(cfg, dtype)
    w = make_model(tmp_path / "big", cfg, seed=37)
    toks = tokens_for(cfg, 620, seed=12)
    want = plain.forward(cfg, w, toks)
    s = Session(tmp_path / "big", device, dtype, pages=40, page_size=16)
    rows = [0, 1, 15, 16, 63, 64, 127, 128, 129, 149, 255, 256, 257, 300, 384, 519]
    got = [s.step(("a", toks[:520], rows)), s.step(("a", toks[520:600], list(range(80))))]
    got += [s.step(("a", [t], [0])) for t in toks[600:]]
    close(np.concatenate(got), np.concatenate([want[rows], want[520:]]), dtype, "larger sizes", rounding_error(tmp_path / "big", device, dtype, toks, want))


def case_greedy_generation_through_the_engine(tmp_path, device, dtype):
    """LLMEngine.generate (scheduler, batching, sampler) against greedy decoding with the plain model."""
    from dli_b200 import LLMEngine, SamplingParams, SchedulerConfig

    cfg = pick("mixed", dtype)
    w = make_model(tmp_path / "g", cfg, seed=31)
    prompts = [tokens_for(cfg, n, seed=60 + n) for n in (5, 19, 1, 11, 8)]
    if device == "cpu":
        from tests import cpu_ops

        model = dli_b200.load_model(tmp_path / "g", dtype, device)
        runner = ModelRunner(model, num_pages=32, page_size=8, max_requests=4, cuda_graphs=False)
        engine = LLMEngine(runner, SchedulerConfig(4, 24), sampler=cpu_ops.CpuSampler())
    else:
        engine = LLMEngine.from_model_dir(tmp_path / "g", dtype=dtype, device=device, num_blocks=32, block_size=8, config=SchedulerConfig(4, 24))
    outs = engine.generate(prompts, SamplingParams(max_tokens=10))
    compared = 0
    for p, got in zip(prompts, outs):
        toks = list(p)
        for t in got:
            row = plain.forward(cfg, w, toks)[-1]
            top = np.sort(row)[-2:]
            if int(np.argmax(row)) != t:
                assert top[1] - top[0] < 2 * TOL[dtype] * max(1.0, np.abs(row).max()), "a generated token differs from the plain model's"
                break
            toks.append(t)
            compared += 1
    assert compared >= 25


CASES = [v for k, v in sorted(globals().items()) if k.startswith("case_")]
