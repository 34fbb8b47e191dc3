"""Cases that compare the engine's Gedunex model with the plain implementation (tests/plain/gedunex_plain.py).

Each case takes (tmp_path, device, dtype) and builds its own small configuration and weights.  The CPU tests run them on
torch stand-ins for the kernels (float32), the GPU tests on the real kernels in both dtypes.  Weights are drawn so that
faults show: forget gates close to one (a lost state changes later tokens), input gates of both signs (the running maximum
moves), sharp attention (one missing key changes the logits), sinks, mixing factors and biases of order one.
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
from tests.plain import gedunex_plain as plain


def attention(heads=4, kv_heads=2, dim=16, vdim=8, scale=0.5, softcap=12.0, window=13, temp=(0.4, 10), v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m}


def memory(heads=3, dim=12, vdim=10, cap=9.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(ff=20, experts=6, top=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, mlps=(), width=48, vocab=89, eps=1e-5, scale=3.0):
    """``mlps``: the layers' feed-forwards, used in turn (None: the layer has none)."""
    mlps = list(mlps) or [moe(), dense()]
    out = {"architecture": "Gedunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": []}
    for i, layer in enumerate(layers):
        out["layers"].append({**layer, "mlp": mlps[i % len(mlps)]})
    return out


# sizes that differ from one another in every respect: head counts that are and are not powers of two, several heads per
# key/value head and one, values shorter and longer than keys, rows that are and are not multiples of 16, with and without
# window, cap, temperature and mixing (the first mixing layer first, later, behind layers that do not mix), a temperature step
# of one token and a broken one, one choice of experts, several, all; dense, routed and absent feed-forwards
CONFIGS = {
    "mixed": config([attention(), memory(), attention(heads=6, kv_heads=1, dim=20, vdim=16, scale=0.3, softcap=7.0, window=21), memory(heads=2, dim=8, vdim=20, cap=15.0),
                     attention(heads=2, kv_heads=2, dim=8, vdim=8, window=5)]),
    "memory_first": config([memory(heads=1, dim=20, vdim=7, cap=4.0), attention(v_mix=False, window=None, temp=None), attention(heads=8, kv_heads=4, dim=16, vdim=24, scale=0.8),
                            attention(heads=4, kv_heads=4, dim=32, vdim=24, softcap=None)], mlps=(None, dense(32), moe(ff=16, experts=4, top=1)), width=40, eps=1e-6),
    "no_mixing": config([attention(v_mix=False), memory(heads=4, dim=16, vdim=16), attention(heads=6, kv_heads=2, dim=64, vdim=40, scale=0.15, softcap=18.0, v_mix=False)],
                        mlps=(moe(ff=64, experts=10, top=4), None), width=64, vocab=130, scale=1.0),
    "only_attention": config([attention(temp=(1.5, 1)), attention(heads=3, kv_heads=1, dim=16, vdim=16, temp=(0.2, 7.5)), attention(heads=12, kv_heads=2, dim=24, vdim=8, window=70)],
                             mlps=(moe(ff=24, experts=5, top=5),), vocab=61),
    "only_memory": config([memory(), memory(heads=2, dim=40, vdim=33, cap=2.0), memory(heads=5, dim=8, vdim=8, cap=30.0)], mlps=(dense(64), None)),
    # nothing a multiple of 4 or 8
    "odd_sizes": config([attention(heads=3, kv_heads=3, dim=7, vdim=5, window=11), memory(heads=3, dim=9, vdim=7), attention(heads=9, kv_heads=3, dim=5, vdim=5, softcap=3.0)],
                        mlps=(moe(ff=11, experts=7, top=3), dense(27)), width=51, vocab=67),
}


def make_model(path: Path, cfg: dict, seed: int = 0, edit=None) -> dict:
    """Writes the folder; returns the tensors as float64 arrays (as stored: values a bfloat16 engine reads unchanged).
    ``edit(tensors)`` may change the tensors before they are written."""
    arch = resolve_architecture(cfg)
    decls = declared_tensors(arch.model_spec(arch.parse_config(cfg)))
    g = torch.Generator().manual_seed(seed)

    def normal(shape, std):
        return torch.randn(shape, generator=g) * std

    def uniform(shape, lo, hi):
        return torch.rand(shape, generator=g) * (hi - lo) + lo

    tensors = {}
    for name, decl in sorted(decls.items()):
        shape = tuple(decl.shape)
        if name.endswith("vmix"):
            t = uniform(shape, 0.3, 0.7)
        elif name.endswith("mix.f.b"):
            t = uniform(shape, 2.0, 5.0)  # the memory keeps most of what it holds
        elif name.endswith("mix.i.b"):
            t = normal(shape, 1.0)
        elif name.endswith("sink"):
            t = normal(shape, 1.0)
        elif name.endswith("router.b"):
            t = normal(shape, 0.5)
        elif name.endswith(".b"):
            t = normal(shape, 0.4)
        elif name.endswith("q.norm") or name.endswith("k.norm"):
            t = 1.3 + normal(shape, 0.3)
        elif len(shape) == 1:
            t = 1.0 + normal(shape, 0.2)
        elif name == "embed":
            t = normal(shape, 1.0)
        elif name.endswith("mix.i") or name.endswith("mix.f"):
            t = normal(shape, 1.5 / shape[1] ** 0.5)
        elif name.endswith("router"):
            t = normal(shape, 2.0 / shape[1] ** 0.5)
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
        if layer.get("mlp") and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
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
    """One layer: each mixer with nothing beside it, with its options one by one; rows of 64 and 128 numbers (which the TMA-fed and
    tcgen05 attention kernels take in bfloat16), of other multiples of 16, and of none; feed-forwards beside the simplest mixer."""
    layers = {
        "plain_softmax": attention(softcap=None, window=None, temp=None, v_mix=False),
        "cap": attention(softcap=2.0, window=None, temp=None, v_mix=False, scale=1.5),
        "window": attention(softcap=None, window=6, temp=None, v_mix=False),
        "temperature": attention(softcap=None, window=None, temp=(2.0, 3), v_mix=False),
        "rows_64": attention(heads=5, kv_heads=1, dim=56, vdim=64, scale=0.2, window=30),
        "rows_64_many_heads": attention(heads=20, kv_heads=1, dim=64, vdim=32, scale=0.2, window=25),
        "rows_128": attention(heads=4, kv_heads=2, dim=128, vdim=120, scale=0.1, window=None),
        "rows_128_capless": attention(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.1, softcap=None),
        "rows_96": attention(heads=3, kv_heads=1, dim=90, vdim=66, scale=0.1),
        "values_longer": attention(heads=2, kv_heads=2, dim=16, vdim=48),
        "memory": memory(),
        "memory_wide": memory(heads=2, dim=136, vdim=40),
        "memory_one_head": memory(heads=1, dim=64, vdim=64, cap=15.0),
        "memory_values_longer": memory(heads=2, dim=16, vdim=72),
        "memory_tiny": memory(heads=7, dim=3, vdim=2),
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
    for name, mlp in {"one_choice": moe(ff=24, experts=4, top=1), "three": moe(ff=16, experts=7, top=3), "all_chosen": moe(ff=8, experts=4, top=4),
                      "many": moe(ff=32, experts=40, top=6), "one_expert": moe(ff=24, experts=1, top=1), "dense_64": dense(64), "dense_odd": dense(21)}.items():
        cfg = config([memory(heads=1, dim=8, vdim=8)], mlps=(mlp,))
        w = make_model(tmp_path / name, cfg, seed=6)
        toks = tokens_for(cfg, 30, seed=3)
        close(Session(tmp_path / name, device, dtype).whole("a", toks), plain.forward(cfg, w, toks), dtype, name)


def case_the_router_s_bias_decides(tmp_path, device, dtype):
    """A bias that lifts one expert above all others makes every token choose it, and enters its weight; another keeps one out."""
    cfg = config([memory(heads=1, dim=8, vdim=8)], mlps=(moe(ff=16, experts=6, top=2),))

    def lift(t):
        t["l0.mlp.router.b"] = torch.tensor([7.0, -12.0, 0.0, 0.0, 0.5, -0.5])

    w = make_model(tmp_path / "r", cfg, seed=8, edit=lift)
    toks = tokens_for(cfg, 25, seed=4)
    ids, weights = plain.route(np.random.default_rng(0).normal(size=(50, 48)), w, "l0.mlp.", cfg["layers"][0]["mlp"]["router"])
    assert (ids[:, 0] == 0).mean() > 0.9 and (ids != 1).all() and weights[:, 0].mean() > 0.9
    close(Session(tmp_path / "r", device, dtype).whole("a", toks), plain.forward(cfg, w, toks), dtype, "routing")


def case_values_are_mixed_with_the_first_mixing_layer_s(tmp_path, device, dtype):
    """Three mixing layers with mixing factors near one behind two that must not be the source: the third's values are nearly the
    first mixing layer's, and leaving that out (or taking another layer's) moves the logits by far more than the tolerance."""
    small = attention(heads=2, kv_heads=1, dim=16, vdim=16, window=9)
    cfg = config([attention(heads=2, kv_heads=1, dim=16, vdim=16, v_mix=False), memory(), small, small, small], mlps=(None,))

    def strong(t):
        for k in t:
            if k.endswith("vmix"):
                t[k] = torch.full_like(t[k], 0.875)

    w = make_model(tmp_path / "v", cfg, seed=12, edit=strong)
    toks = tokens_for(cfg, 40, seed=9)
    want = plain.forward(cfg, w, toks)
    off = {k: np.zeros_like(v) if k.endswith("vmix") else v for k, v in w.items()}
    assert np.abs(plain.forward(cfg, off, toks) - want).max() > 0.5
    s = Session(tmp_path / "v", device, dtype)
    got = [s.step(("a", toks[:25], list(range(25)))), s.step(("a", toks[25:28], [0, 1, 2]))] + [s.step(("a", [t], [0])) for t in toks[28:]]
    close(np.concatenate(got), want, dtype, "mixed values")


def case_prefill_then_token_by_token(tmp_path, device, dtype):
    """A prompt in one step, then 60 tokens one at a time (the windows pass over decoded tokens), against the whole sequence at once;
    and a sequence fed token by token from its very first token."""
    cfg = pick("mixed", dtype)
    w = make_model(tmp_path / "m", cfg, seed=7)
    toks = tokens_for(cfg, 95, seed=3)
    want = plain.forward(cfg, w, toks)
    s = Session(tmp_path / "m", device, dtype, pages=40)
    got = [s.step(("a", toks[:35], list(range(35))))]
    got += [s.step(("a", [t], [0])) for t in toks[35:]]
    close(np.concatenate(got), want, dtype, "prompt then decode", rounding_error(tmp_path / "m", device, dtype, toks, want))
    s.free("a")
    got = [s.step(("b", [t], [0])) for t in toks[:20]]
    close(np.concatenate(got), want[:20], dtype, "token by token from the start")


def case_long_decoding(tmp_path, device, dtype):
    """A short prompt and 300 decoded tokens: the memory is carried through hundreds of steps, pages behind the windows are given
    back, the temperature steps up thirty times."""
    cfg = config([memory(heads=2, dim=16, vdim=16, cap=15.0), attention(heads=2, kv_heads=1, dim=16, vdim=8, window=21), memory(heads=1, dim=8, vdim=8)],
                 mlps=(moe(ff=16, experts=4, top=2),), width=32)
    cfg = steady(cfg, dtype)

    def lasting(t):
        for k in t:
            if k.endswith("mix.f.b"):
                t[k] = torch.full_like(t[k], 6.5)

    w = make_model(tmp_path / "l", cfg, seed=9, edit=lasting)
    toks = tokens_for(cfg, 310, seed=4)
    want = plain.forward(cfg, w, toks)
    s = Session(tmp_path / "l", device, dtype, pages=44, page_size=8)
    s.step(("a", toks[:10], []))
    got = np.concatenate([s.step(("a", [t], [0])) for t in toks[10:]])
    close(got, want[10:], dtype, "long decoding", rounding_error(tmp_path / "l", device, dtype, toks, want))
    other = list(toks)
    other[:40] = tokens_for(cfg, 40, seed=400)
    assert np.abs(plain.forward(cfg, w, other)[-1] - want[-1]).max() > 0.02, "the memory does not last long enough for this test"


def case_portions_of_many_sizes(tmp_path, device, dtype):
    """Portions down to two tokens and single tokens between them, cut inside pages, windows and tiles of tokens, and portions longer
    than a tile of the matrix memory's tensor-core kernel, whose last tile is not full."""
    for name in ("mixed", "memory_first", "no_mixing", "odd_sizes", "only_memory"):
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


def case_pages_and_slots_used_again(tmp_path, device, dtype):
    """A pool for two short requests and two state slots: request after request takes the pages and the slot a finished one gave
    back, and computes what it would compute in a fresh engine."""
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


def _quiet_sink(t):
    """No sink, and mixer outputs as large as the embedding (whose large scale keeps the positions out of the choice of keys)."""
    for k in t:
        if k.endswith("sink"):
            t[k] = torch.full_like(t[k], -30.0)
        if k.endswith("mix.o"):
            t[k] = t[k] * 300.0


def _pair(cfg, w):
    """In a model of one attention layer with a large embedding scale a raw score depends nearly on the two tokens alone.  Returns a
    token whose last head (the one with the smallest slope) scores one other token's key far above every other's, that token, and
    tokens whose keys it scores far below."""
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    h = plain.rms_unit(w["embed"], eps) * w["l0.norm1"]
    q = (plain.rms_unit(h @ w["l0.mix.q"].T + w["l0.mix.q.b"], eps) * w["l0.mix.q.norm"])[:, -m["dim"] :]
    k = (plain.rms_unit(h @ w["l0.mix.k"].T + w["l0.mix.k.b"], eps) * w["l0.mix.k.norm"])[:, -m["dim"] :]
    s = q @ k.T * m["scale"]
    s = m["softcap"] * np.tanh(s / m["softcap"])
    V = cfg["vocab"]
    gap = np.sort(s, 1)[:, -1] - np.median(s, 1)
    asker = int(max((t for t in range(V) if s[t].argmax() != t), key=lambda t: gap[t]))
    key = int(s[asker].argmax())
    noise = [t for t in range(V) if s[asker, t] < s[asker, key] - 10 and t != asker]
    assert len(noise) > 15
    return asker, key, noise


FAR = dict(heads=2, kv_heads=1, dim=16, vdim=16, scale=4.0, softcap=30.0, temp=(0.05, 40))


def case_one_far_key_decides(tmp_path, device, dtype):
    """Sequences made so that the last token's last head puts nearly all its mass on ONE key among hundreds — at a page border,
    beside one, at the very start: a kernel that skips or misplaces that key changes the logits by far more than the tolerance.  In
    a prompt and decoded, with rows of 16 and of 64 numbers (the other attention kernels)."""
    for rows in (16, 64):
        cfg = config([attention(**{**FAR, "vdim": rows}, window=None)], mlps=(None,), width=32, vocab=50, scale=300.0)
        w = make_model(tmp_path / f"far{rows}", cfg, seed=19, edit=_quiet_sink)
        asker, key, noise = _pair(cfg, w)
        s = Session(tmp_path / f"far{rows}", device, dtype, pages=48, page_size=8)
        for far in (8, 15, 16, 1, 0, 100, 263):
            toks = [noise[i] for i in np.random.default_rng(far).integers(0, len(noise), 330)]
            toks[far], toks[-1] = key, asker
            want = plain.forward(cfg, w, toks)
            without = list(toks)
            without[far] = noise[0]
            assert np.abs(plain.forward(cfg, w, without)[-1] - want[-1]).max() > 0.5, "the far key does not matter enough for this test"
            close(s.whole("p", toks)[-1], want[-1], dtype, f"rows of {rows}: far key {far} in a prompt")
            s.free("p")
            s.step(("d", toks[:-1], []))
            close(s.step(("d", toks[-1:], [0]))[0], want[-1], dtype, f"rows of {rows}: far key {far} decoded")
            s.free("d")


def case_one_key_at_the_window_s_edge(tmp_path, device, dtype):
    """The same construction with windows: the deciding key sits on the last place the window still holds (it decides), and one
    place further back (it must not be seen); in a prompt, decoded alone and inside a last portion, with the window's edge inside a
    page and on a page border; windows of 24 and, with rows of 64 numbers, of 130 keys (over a tile of keys)."""
    for window, rows, lengths in ((24, 16, (60, 57)), (130, 64, (200, 257))):
        cfg = config([attention(**{**FAR, "vdim": rows}, window=window)], mlps=(None,), width=32, vocab=50, scale=300.0)
        w = make_model(tmp_path / f"edge{window}", cfg, seed=19, edit=_quiet_sink)
        asker, key, noise = _pair(cfg, w)
        s = Session(tmp_path / f"edge{window}", device, dtype, pages=40, page_size=8)
        for length in lengths:
            last = length - 1
            logits = {}
            for name, place in (("inside", last - window + 1), ("outside", last - window)):
                toks = [noise[i] for i in np.random.default_rng(length).integers(0, len(noise), length)]
                toks[place], toks[last] = key, asker
                want = plain.forward(cfg, w, toks)
                logits[name] = want[-1]
                close(s.whole("p", toks)[-1], want[-1], dtype, f"key {name} the window of {window}, prompt of {length}")
                s.free("p")
                s.step(("d", toks[:-1], []))
                close(s.step(("d", toks[-1:], [0]))[0], want[-1], dtype, f"key {name} the window of {window}, decoded at {last}")
                s.free("d")
                s.step(("c", toks[: last - 5], []))
                close(s.step(("c", toks[last - 5 :], [5]))[0], want[-1], dtype, f"key {name} the window of {window}, in a last portion of 6")
                s.free("c")
            assert np.abs(logits["inside"] - logits["outside"]).max() > 0.5, "the key at the window's edge does not matter enough for this test"


def case_a_sink_takes_the_mass(tmp_path, device, dtype):
    """Sinks far above every score in some heads and far below in others: the first heads' outputs all but vanish, the others' do not
    notice; left out, the logits move by far more than the tolerance.  A sink is neither capped (it lies above the cap) nor
    charged for distance."""
    cfg = config([attention(heads=4, kv_heads=2, dim=16, vdim=16, softcap=5.0, window=11)], mlps=(None,), width=32, vocab=40)

    def sinks(t):
        t["l0.mix.sink"] = torch.tensor([12.0, -12.0, 3.0, 0.0])

    w = make_model(tmp_path / "sink", cfg, seed=29, edit=sinks)
    toks = tokens_for(cfg, 40, seed=8)
    want = plain.forward(cfg, w, toks)
    none = {k: np.full_like(v, -1e9) if k.endswith("sink") else v for k, v in w.items()}
    assert np.abs(plain.forward(cfg, none, toks) - want).max() > 0.3
    s = Session(tmp_path / "sink", device, dtype)
    got = [s.step(("a", toks[:30], list(range(30))))] + [s.step(("a", [t], [0])) for t in toks[30:]]
    close(np.concatenate(got), want, dtype, "sink")


def case_one_write_lasts_in_the_memory(tmp_path, device, dtype):
    """Input gates that are shut for every token but one, and forget gates that stay open: what that token wrote is read 200 tokens
    later (at the start, at a tile's last and first place, inside it), across prompts, portions and decoding."""
    cfg = config([memory(heads=2, dim=16, vdim=16, cap=15.0)], mlps=(None,), width=32, vocab=50, scale=300.0)
    special = 7

    def gates(t):
        t["l0.mix.f"] = torch.zeros_like(t["l0.mix.f"])
        t["l0.mix.f.b"] = torch.full_like(t["l0.mix.f.b"], 30.0)
        e = t["embed"][special]
        direction = e / e.norm()
        t["embed"] = t["embed"] - torch.outer(t["embed"] @ direction, direction) * 1.0
        t["embed"][special] = e
        t["l0.norm1"] = torch.ones_like(t["l0.norm1"])
        t["l0.mix.i"] = (direction * 4.0).repeat(2, 1)
        t["l0.mix.i.b"] = torch.full_like(t["l0.mix.i.b"], -9.0)
        t["l0.mix.o"] = t["l0.mix.o"] * 300.0  # as large as the embedding, whose large scale keeps the positions out of the gates

    w = make_model(tmp_path / "write", cfg, seed=33, edit=gates)
    s = Session(tmp_path / "write", device, dtype, pages=40, page_size=8)
    for place in (0, 1, 63, 64, 70):
        toks = [t if t != special else 8 for t in tokens_for(cfg, 270, seed=50 + place)]
        toks[place] = special
        want = plain.forward(cfg, w, toks)
        without = list(toks)
        without[place] = 9
        assert np.abs(plain.forward(cfg, w, without)[-1] - want[-1]).max() > 0.3, "the write does not last enough for this test"
        close(s.whole("p", toks), want, dtype, f"write at {place}, prompt")
        s.free("p")
        got = [s.step(("c", toks[:100], list(range(100)))), s.step(("c", toks[100:103], [0, 1, 2])), s.step(("c", toks[103:250], list(range(147))))]
        got += [s.step(("c", [t], [0])) for t in toks[250:]]
        close(np.concatenate(got), want, dtype, f"write at {place}, portions and decoding")
        s.free("c")


def case_the_first_tokens(tmp_path, device, dtype):
    """Sequences of one, two and three tokens, and a first step of one token followed by portions: a memory that starts at zero with
    its maximum at zero (input gates far below zero show it), windows and pages that are not full."""
    cfg = pick("mixed", dtype)

    def shut(t):
        for k in t:
            if k.endswith("mix.i.b"):
                t[k] = torch.full_like(t[k], -4.0)

    w = make_model(tmp_path / "m", cfg, seed=27, edit=shut)
    s = Session(tmp_path / "m", device, dtype)
    for n in (1, 2, 3):
        toks = tokens_for(cfg, n, seed=70 + n)
        close(s.whole("a", toks), plain.forward(cfg, w, toks), dtype, f"{n} tokens")
        s.free("a")
    toks = tokens_for(cfg, 32, seed=75)
    got = np.concatenate([s.step(("b", toks[:1], [0])), s.step(("b", toks[1:3], [0, 1])), s.step(("b", toks[3:], list(range(29))))])
    close(got, plain.forward(cfg, w, toks), dtype, "one token, then portions")


def case_layer_sizes_of_a_larger_model(tmp_path, device, dtype):
    """Memory heads of 128 x 128 and attention rows of 128 and 64 numbers (which the TMA-fed and tcgen05 kernels take in bfloat16,
    with several tiles of queries and keys), a prompt of 600 tokens in two portions (many tokens per expert; the products for many
    tokens), then decoding."""
    cfg = config([attention(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.06, softcap=25.0, window=150), memory(heads=3, dim=128, vdim=128, cap=15.0),
                  attention(heads=16, kv_heads=4, dim=64, vdim=64, scale=0.1, softcap=25.0, window=300, v_mix=True)],
                 mlps=(dense(512), moe(ff=128, experts=8, top=2)), width=256, vocab=300, scale=5.0)
    cfg = steady(cfg, dtype)
    w = make_model(tmp_path / "big", cfg, seed=37)
    toks = tokens_for(cfg, 620, seed=12)
    want = plain.forward(cfg, w, toks)
    s = Session(tmp_path / "big", device, dtype, pages=40, page_size=16)
    rows = [0, 1, 15, 16, 63, 64, 127, 128, 129, 149, 150, 151, 299, 300, 301, 519]
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
