"""The kernels that came with the one-norm parallel layer — sinusoidal embedding, whole-projection norm with temperature and mixed
values, bent attention scores, the matrix memory, the router by softmax over the chosen — against plain PyTorch float32
restatements (tests/cpu_ops.py), in float32 and bfloat16, at sizes that take the 16-byte paths and sizes that do not."""

import pytest
import torch

from dli_b200.kernels import ops
from tests import cpu_ops as ref

pytestmark = pytest.mark.gpu

DTYPES = [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)]


def _rand(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(*shape, generator=g) * scale


def _close(got, want, tol, what=""):
    got, want = got.float().cpu(), want.float()
    err = (got - want).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), f"{what}: max error {err}"


def _i32(values):
    return torch.tensor(values, dtype=torch.int32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H", [1, 40, 77, 256, 2050])
def test_sinusoid_embedding(dtype, H):
    """Also positions far out: the angles keep float32's precision."""
    table, ids = _rand(30, H, seed=1).to(dtype), _i32([3, 29, 0, 7, 7])
    pos = _i32([0, 1, 95, 4097, 60001])
    freq = torch.tensor([10000.0 ** (-2.0 * i / H) for i in range((H + 1) // 2)], dtype=torch.float64)
    head = freq.float()
    parts = torch.stack([head, (freq - head.double()).float()])
    want, got = torch.empty(5, H), torch.empty(5, H, device="cuda")
    ref.sinusoid_embedding(want, table, 2.5, parts, ids, pos)
    ang = pos.double()[:, None] * freq[None, :]
    exact = table[ids.long()].double() * 2.5 + torch.stack([ang.sin(), ang.cos()], -1).reshape(5, -1)[:, :H]
    ops.sinusoid_embedding(got, table.cuda(), 2.5, parts.cuda(), ids.cuda(), pos.cuda())
    assert (got.cpu().double() - exact).abs().max() < 2e-6


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 1, 16, 8, 16), (3, 3, 10, 7, 10), (8, 2, 64, 48, 64), (2, 1, 24, 40, 48), (2, 2, 128, 128, 128), (20, 1, 64, 64, 64)])
def test_qk_norm_mix_store(dtype, tol, sizes):
    nh, nkv, d, dv, D = sizes
    n, page, pages = 7, 4, 6
    cols = (nh + nkv) * d + nkv * dv
    pos, slots = _i32([0, 1, 2, 300, 31, 5, 1000]), _i32([20, 1, 7, 3, 12, 13, 23])
    wq, wk, bias = 1 + 0.3 * _rand(nh * d, seed=2), 1 + 0.3 * _rand(nkv * d, seed=3), _rand(cols, seed=4)
    for in_dtype in {dtype, torch.float32}:
        x = _rand(n, cols, seed=1).to(in_dtype)
        for eps, temp, mix, with_bias in ((1e-5, (0.3, 8.0), "mix", True), (1e-5, (0.0, 1.0), "source", False), (None, (0.7, 2.5), None, True)):
            source = _rand(n, nkv * dv, seed=5) if mix == "mix" else (torch.zeros(n, nkv * dv) if mix else None)
            lam = 0.4 if mix == "mix" else None
            outs = []
            for module, where in ((ref, "cpu"), (ops, "cuda")):
                q = torch.full((n, nh * D), 9.0, dtype=dtype, device=where)
                pools = [torch.full((pages, nkv, page, D), 9.0, dtype=dtype, device=where) for _ in range(2)]
                src = None if source is None else source.clone().to(where)
                module.qk_norm_mix_store(q, x.to(where), bias.to(where) if with_bias else None, wq.to(where), wk.to(where), eps, pos.to(where), temp, src, lam,
                                         slots.to(where), pools[0], pools[1], nh, nkv, d, dv, page)
                outs.append((q, *pools) + (() if src is None else (src,)))
            for got, want, name in zip(outs[1], outs[0], ("q", "k", "v", "source")):
                _close(got, want, tol if name != "source" else 1e-6, f"{name} {in_dtype} {mix}")


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_group_norm_with_divisors(dtype, tol):
    n = 9
    for inner, parts in ((48, 3), (256, 2), (35, 5), (2048, 16)):
        y, z, wt = _rand(n, inner, seed=4) * 3, _rand(n, inner, seed=5).to(dtype), 1 + 0.2 * _rand(inner, seed=6)
        div = torch.rand(n, parts, generator=torch.Generator().manual_seed(7)) * 50 + 1e-3  # the norm's eps sees it
        want, got = torch.empty(n, inner, dtype=dtype), torch.empty(n, inner, dtype=dtype, device="cuda")
        ref.gated_group_rmsnorm(want, y, z, 0, wt, parts, 0.01, gate_after=True, gate="sigmoid", divisor=div)
        ops.gated_group_rmsnorm(got, y.cuda(), z.cuda(), 0, wt.cuda(), parts, 0.01, gate_after=True, gate="sigmoid", divisor=div.cuda())
        _close(got, want, tol, f"{inner} / {parts}")


def _memory_inputs(dtype, heads, d, dv, n, seed=7):
    g = torch.Generator().manual_seed(seed)
    u = torch.randn(n, heads * (2 * d + 2 * dv), generator=g).to(dtype)
    gates = torch.randn(n, 2 * heads, generator=g) * 4
    bias = torch.randn(2 * heads, generator=g)
    bias[heads:] += 4.0
    state = torch.randn(5, heads, dv + 1, d, generator=g) * 0.5
    top = (torch.rand(5, heads, 1, generator=g) * 3).expand(5, heads, dv + 1).contiguous()
    return u, gates, bias, state, top


@pytest.mark.parametrize("form", ["walk", "chunk"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(4, 12, 10), (2, 32, 32), (3, 9, 7), (2, 48, 56), (2, 128, 128), (1, 136, 40), (2, 64, 63), (1, 256, 48), (2, 16, 130), (1, 24, 15), (1, 40, 16)])
def test_matrix_memory(sizes, dtype, form):
    """Portions of 1, 70, 3, 128 and 33 tokens from states that are not zero, in scattered slots; the state afterwards; then the
    same tokens one at a time.  Both forms are float32 in effect, whatever the inputs' dtype: the tolerances are float32's."""
    heads, d, dv = sizes
    if form == "chunk" and dtype != torch.bfloat16:
        pytest.skip("the tensor-core form takes bfloat16")
    lens = (1, 70, 3, 128, 33)
    n = sum(lens)
    u, gates, bias, state, top = _memory_inputs(dtype, heads, d, dv, n)
    q_start = _i32([0] + torch.tensor(lens).cumsum(0).tolist())
    slots = _i32([3, 0, 4, 1, 2])

    def run(module, where, form=None, one_by_one=False, **more):
        o, div = torch.zeros(n, heads * dv, device=where), torch.zeros(n, heads, device=where)
        s, m = state.clone().to(where), top.clone().to(where)
        ud, gd, bd = u.to(where), gates.to(where), bias.to(where)
        if not one_by_one:
            module.matrix_memory_scan(o, div, ud, gd, bd, 9.0, s, m, q_start.to(where), slots.to(where), max_len=max(lens), **({"form": form} if form else {}), **more)
        else:
            for i in range(max(lens)):  # the i-th token of every sequence that has one
                seqs = [k for k, L in enumerate(lens) if i < L]
                rows = torch.tensor([int(q_start[k]) + i for k in seqs], device=where)
                oo, dd = torch.zeros(len(seqs), heads * dv, device=where), torch.zeros(len(seqs), heads, device=where)
                module.matrix_memory_scan(oo, dd, ud[rows].contiguous(), gd[rows].contiguous(), bd, 9.0, s, m, _i32(range(len(seqs) + 1)).to(where),
                                          slots[seqs].to(where), max_len=1)
                o[rows], div[rows] = oo, dd
        return o, div, s, m

    want = run(ref, "cpu")
    for more in ({},) if form == "walk" else ({}, {"segments": 1}, {"segments": 2}, {"segments": 7}):  # (seven: more than a sequence has tiles)
        for a, b, what in zip(run(ops, "cuda", form, **more), want, ("o", "divisor", "state", "top")):
            _close(a, b, 2e-5, f"{what} {more}")
    if form == "walk":
        for a, b, what in zip(run(ops, "cuda", one_by_one=True), want, ("o", "divisor", "state", "top")):
            _close(a, b, 2e-5, f"token by token: {what}")


def test_matrix_memory_with_gates_at_their_extremes():
    """Forget gates that forget nearly everything and input gates that swing over the whole cap: the weights of a tile span a
    hundred powers of e, and nothing overflows."""
    heads, d, dv, n = 2, 32, 32, 200
    u, gates, bias, state, top = _memory_inputs(torch.bfloat16, heads, d, dv, n)
    gates = gates * 20
    gates[50:120, heads:] = -60.0
    q_start, slots = _i32([0, n]), _i32([2])
    out = []
    for module, where, more in ((ref, "cpu", {}), (ops, "cuda", {"segments": 1}), (ops, "cuda", {"segments": 3}), (ops, "cuda", {"form": "walk"})):
        o, div = torch.zeros(n, heads * dv, device=where), torch.zeros(n, heads, device=where)
        s, m = state.clone().to(where), top.clone().to(where)
        module.matrix_memory_scan(o, div, u.to(where), gates.to(where), bias.to(where), 15.0, s, m, q_start.to(where), slots.to(where), max_len=n, **more)
        out.append((o.view(n, heads, dv) / div[:, :, None], m, s))
    for got in out[1:]:
        for a, b, what in zip(got, out[0], ("o / divisor", "top", "state")):
            assert torch.isfinite(a).all()
            _close(a, b, 1e-3, what)


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_router_by_softmax_over_the_chosen(dtype, tol):
    for W, E, top in ((48, 6, 2), (64, 13, 3), (50, 7, 7), (128, 40, 6), (256, 16, 1), (32, 1, 1)):
        router, bias = _rand(E, W, seed=1, scale=2.0 / W**0.5), _rand(E, seed=2)
        for n in (1, 5, 300):
            x = _rand(n, W, seed=10 + n).to(dtype)
            ids_ref, w_ref = torch.zeros(n, top, dtype=torch.int32), torch.zeros(n, top)
            ids_dev, w_dev = ids_ref.cuda(), w_ref.cuda()
            ref.moe_route(ids_ref, w_ref, x, router, bias, 1, 1, 1.0, "softmax_chosen")
            ops.moe_route(ids_dev, w_dev, x.cuda(), router.cuda(), bias.cuda(), 1, 1, 1.0, "softmax_chosen")
            same = (ids_dev.cpu() == ids_ref).all(1)
            assert same.float().mean() > 0.97, "routing differs on more than near ties"
            _close(w_dev.cpu()[same], w_ref[same], 1e-5, "weights")
            assert (w_dev.sum(1) - 1).abs().max() < 1e-5


def _paged_batch(nh, nkv, d, dtype, page, lens, kv, seed):
    """Scrambled pages (unused ones poisoned), a batch of single tokens and portions; returns what the attention entry takes."""
    g = torch.Generator().manual_seed(seed)
    need = [-(-L // page) for L in kv]
    pages = sum(need) + 4
    k_pool, v_pool = (torch.randn(pages, nkv, page, d, generator=g) * 0.5).to(dtype), torch.randn(pages, nkv, page, d, generator=g).to(dtype)
    perm = torch.randperm(pages, generator=g)
    tables = torch.full((len(kv), max(need) + 2), -1, dtype=torch.int32)
    at = 0
    for s, c in enumerate(need):
        tables[s, :c] = perm[at : at + c].to(torch.int32)
        at += c
    k_pool[perm[at:]] = float("nan")
    v_pool[perm[at:]] = float("nan")
    n = sum(lens)
    q = torch.randn(n, nh * d, generator=g).to(dtype)
    q_start = _i32([0] + torch.tensor(lens).cumsum(0).tolist())
    seq_of = torch.cat([torch.full((L,), s, dtype=torch.int32) for s, L in enumerate(lens)])
    pos = torch.cat([torch.arange(K - L, K, dtype=torch.int32) for K, L in zip(kv, lens)])
    singles = sum(L == 1 for L in lens)

    class Group:
        block_tables, slots = tables.cuda(), None

    class Batch:
        num_single, num_seqs, max_q_len, max_kv_len = singles, len(lens), max(lens), max(kv)
        max_kv_len_single = max(K for K, L in zip(kv, lens) if L == 1)
        launch_keys = {}

        def group(self, i):
            return Group

    Batch.q_start, Batch.kv_len, Batch.seq_of_token, Batch.positions = q_start.cuda(), _i32(kv).cuda(), seq_of.cuda(), pos.cuda()

    class Cache:
        k, v, page_size, group = k_pool.cuda(), v_pool.cuda(), page, 0

    return q, k_pool, v_pool, tables, seq_of, pos, Batch, Cache


@pytest.mark.parametrize("bend", ["cap and slopes", "slopes", "cap"])
@pytest.mark.parametrize("window", [None, 64, 150])
@pytest.mark.parametrize("dtype,d,heads", [(torch.float32, 24, (4, 2)), (torch.bfloat16, 48, (4, 2)), (torch.bfloat16, 64, (5, 1)), (torch.bfloat16, 64, (20, 1)),
                                           (torch.bfloat16, 96, (6, 3)), (torch.bfloat16, 128, (4, 2)), (torch.bfloat16, 128, (3, 3)), (torch.bfloat16, 20, (2, 1))])
def test_bent_scores_in_every_attention_kernel(dtype, d, heads, window, bend):
    """A soft cap that bites, slopes from steep to nearly flat, a sink per head, over portions and single tokens, with and without
    split keys: the CUDA-core, mma.sync, TMA decode and tcgen05 prefill kernels (one and two query tiles)."""
    from dli_b200.kernels import attention as attn

    nh, nkv = heads
    q, k_pool, v_pool, tables, seq_of, pos, Batch, Cache = _paged_batch(nh, nkv, d, dtype, 16, [1, 1, 1, 5, 70, 300], [150, 37, 1, 61, 70, 430], seed=d + nh)
    g = torch.Generator().manual_seed(3)
    sinks = torch.randn(nh, generator=g)
    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / nh) for h in range(nh)]) if "slopes" in bend else None
    cap = 3.0 if "cap" in bend else None
    n, scale = q.shape[0], 4.0 / d**0.5
    want = torch.zeros(n, nh * d, dtype=dtype)
    ref.paged_attention_simt(want, q, torch.nan_to_num(k_pool), torch.nan_to_num(v_pool), tables, seq_of, pos, nh, scale, window, sinks, cap, slopes)
    for splits in (None, 2, 4):
        got = torch.zeros(n, nh * d, dtype=dtype, device="cuda")
        attn.paged_attention(got, q.cuda(), Cache, Batch(), nh, scale, window, splits=splits, sink=sinks.cuda(), softcap=cap,
                             slopes=None if slopes is None else slopes.cuda())
        _close(got, want, 2e-5 if dtype == torch.float32 else 3e-2, f"splits={splits}")


@pytest.mark.parametrize("d", [64, 128])
def test_bent_decode_with_eight_warps_and_many_splits(d):
    """A long context for one sequence: eight warps a CTA at rows of 64, sixteen splits in a cluster, and splits merged by the second
    kernel."""
    from dli_b200.kernels import attention as attn

    nh, nkv = 8, 2
    q, k_pool, v_pool, tables, seq_of, pos, Batch, Cache = _paged_batch(nh, nkv, d, torch.bfloat16, 16, [1], [9000], seed=5)
    slopes = torch.tensor([0.5, 0.1, 0.02, 0.004, 0.001, 0.0002, 0.0, 0.3])
    want = torch.zeros(1, nh * d, dtype=torch.bfloat16)
    ref.paged_attention_simt(want, q, torch.nan_to_num(k_pool), torch.nan_to_num(v_pool), tables, seq_of, pos, nh, 0.4, None, None, 6.0, slopes)
    for splits in (1, 8, 16, 24):
        got = torch.zeros(1, nh * d, dtype=torch.bfloat16, device="cuda")
        attn.paged_attention(got, q.cuda(), Cache, Batch(), nh, 0.4, None, splits=splits, softcap=6.0, slopes=slopes.cuda())
        _close(got, want, 2e-2, f"splits={splits}")


def test_plain_libraries_refuse_bent_scores():
    """The libraries without the instructions say so instead of leaving the scores as they are."""
    from ctypes import c_float, c_int, c_longlong, c_void_p

    f = ops._fn("attention_tc.cu", "dli_paged_decode_tma", [c_void_p, c_void_p, c_longlong, c_void_p, c_void_p, c_longlong, c_void_p, c_int, c_void_p, c_void_p]
                + [c_int] * 9 + [c_float, c_float, c_void_p, c_float, c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p])
    none = c_void_p(0)
    assert f(none, none, 0, none, none, 0, none, 0, none, none, 0, 1, 0, 1, 1, 64, 64, 16, 0, 1.0, 0.0, none, 5.0, none, 1, none, none, 0, none) == 1001
