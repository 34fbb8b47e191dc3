"""The kernels that came or grew with the output-norm attention design — norms per head and per projection with rotation and values of
their own size, every attention kernel with keys and values of different sizes, the router by softmax over all outputs, experts without
a gate, identities, a shared feed-forward — against plain PyTorch float32 restatements (tests/cpu_ops.py), in float32 and
bfloat16, at sizes that take the 16-byte paths and sizes that do not."""

import pytest
import torch

from dli_b200.kernels import attention as attn
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


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("norm", ["head", "projection", None])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 8, 16, 8, 8), (3, 3, 7, 5, 7, 5, 6), (6, 2, 64, 40, 64, 48, 64), (4, 1, 72, 104, 80, 112, 16), (2, 2, 24, 24, 32, 32, 24),
                                   (5, 1, 40, 16, 48, 16, 0), (2, 1, 128, 64, 128, 64, 32), (40, 8, 128, 128, 128, 128, 128), (3, 1, 11, 9, 16, 16, 4), (2, 1, 256, 8, 256, 8, 16)])
def test_qk_norm_rotary_store(dtype, tol, norm, sizes):
    """Rows padded with zeros, values of another size, with and without the write of keys and values (a layer that reads another's)."""
    nh, nkv, d, dv, row, vrow, rot = sizes
    n, page, pages = 7, 4, 6
    cols = (nh + nkv) * d + nkv * dv
    pos, slots = _i32([0, 1, 2, 300, 31, 5, 1000]), _i32([20, 1, 7, 3, 12, 13, 23])
    inv = torch.tensor([900.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)]) if rot else None
    per_head = norm == "head"
    wq, wk = (None, None) if norm is None else (1 + 0.3 * _rand((1 if per_head else nh) * d, seed=2), 1 + 0.3 * _rand((1 if per_head else nkv) * d, seed=3))
    for write in (True, False):
        x = _rand(n, cols if write else nh * d, seed=1).to(dtype)
        outs = []
        for module, where in ((ref, "cpu"), (ops, "cuda")):
            pools = [torch.full((pages, nkv, page, r), 9.0, dtype=dtype, device=where) for r in (row, vrow)]

            def dev(t):
                return None if t is None else t.to(where)

            q = module.qk_norm_rotary_store(dev(x), dev(wq), dev(wk) if write else None, 1e-5, dev(pos), dev(inv), dev(slots) if write else None,
                                            pools[0] if write else None, pools[1] if write else None, nh, nkv, d, rot, page, write, False, value_dim=dv,
                                            per_head=per_head, row=row)
            outs.append((q, *pools))
        for got, want, name in zip(outs[1], outs[0], ("q", "k", "v")):
            _close(got, want, tol, f"{name}, write={write}")


def _paged_batch(nh, nkv, d, dv, dtype, page, lens, kv, seed):
    """Scrambled pages (unused ones poisoned), a batch of single tokens and portions; returns what the attention entry takes."""
    g = torch.Generator().manual_seed(seed)
    need = [-(-L // page) for L in kv]
    pages = sum(need) + 4
    k_pool, v_pool = (torch.randn(pages, nkv, page, d, generator=g) * 0.5).to(dtype), torch.randn(pages, nkv, page, dv, generator=g).to(dtype)
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
        max_kv_len_single = max((K for K, L in zip(kv, lens) if L == 1), default=0)
        launch_keys = {}

        def group(self, i):
            return Group

    Batch.q_start, Batch.kv_len, Batch.seq_of_token, Batch.positions = q_start.cuda(), _i32(kv).cuda(), seq_of.cuda(), pos.cuda()

    class Cache:
        k, v, page_size, group = k_pool.cuda(), v_pool.cuda(), page, 0

    return q, k_pool, v_pool, tables, seq_of, pos, Batch, Cache


SIZES = [(64, 128), (128, 64), (72, 40), (40, 104), (96, 96), (48, 48), (112, 88), (64, 16), (8, 64), (128, 80), (80, 128), (16, 48), (160, 48), (24, 144), (20, 28), (256, 32), (16, 256)]


@pytest.mark.parametrize("sink", [None, 0.0])
@pytest.mark.parametrize("d,dv", SIZES)
def test_attention_with_values_of_their_own_size(d, dv, sink):
    """Portions and single tokens over scrambled pages, with and without split keys, in bfloat16: the TMA decode and tcgen05 prefill kernels
    with whole and with partly filled slabs, the mma.sync kernels, and the CUDA-core kernel for the sizes that only it takes."""
    for nh, nkv, page, window in ((4, 2, 16, None), (3, 3, 8, None), (20, 1, 32, None), (4, 2, 16, 90)):
        q, k_pool, v_pool, tables, seq_of, pos, Batch, Cache = _paged_batch(nh, nkv, d, dv, torch.bfloat16, page, [1, 1, 1, 5, 70, 300], [150, 37, 1, 61, 70, 430], seed=d + nh)
        n, scale = q.shape[0], 4.0 / d**0.5
        want = torch.zeros(n, nh * dv, dtype=torch.bfloat16)
        ref.paged_attention_simt(want, q, torch.nan_to_num(k_pool), torch.nan_to_num(v_pool), tables, seq_of, pos, nh, scale, window, sink)
        for splits in (None, 2, 4):
            got = torch.full((n, nh * dv), 7.0, dtype=torch.bfloat16, device="cuda")
            attn.paged_attention(got, q.cuda(), Cache, Batch(), nh, scale, window, splits=splits, sink=sink)
            _close(got, want, 3e-2, f"{nh} heads on {nkv}, pages of {page}, window {window}, splits={splits}")


@pytest.mark.parametrize("d,dv", [(64, 128), (20, 28), (7, 33), (300, 12)])
def test_float32_attention_with_values_of_their_own_size(d, dv):
    nh, nkv = 6, 2
    q, k_pool, v_pool, tables, seq_of, pos, Batch, Cache = _paged_batch(nh, nkv, d, dv, torch.float32, 16, [1, 1, 5, 70], [150, 1, 61, 70], seed=d)
    want, got = torch.zeros(q.shape[0], nh * dv), torch.zeros(q.shape[0], nh * dv, device="cuda")
    ref.paged_attention_simt(want, q, torch.nan_to_num(k_pool), torch.nan_to_num(v_pool), tables, seq_of, pos, nh, 3.0 / d**0.5, None, 0.0)
    attn.paged_attention(got, q.cuda(), Cache, Batch(), nh, 3.0 / d**0.5, None, sink=0.0)
    _close(got, want, 2e-5)


@pytest.mark.parametrize("d,dv", [(128, 64), (64, 128), (72, 40), (96, 128)])
def test_many_splits_with_values_of_their_own_size(d, dv):
    """A long context for one sequence: splits merged in a cluster of 16, of 8, and by the second kernel."""
    nh, nkv = 8, 2
    q, k_pool, v_pool, tables, seq_of, pos, Batch, Cache = _paged_batch(nh, nkv, d, dv, torch.bfloat16, 16, [1], [9000], seed=5)
    want = torch.zeros(1, nh * dv, dtype=torch.bfloat16)
    ref.paged_attention_simt(want, q, torch.nan_to_num(k_pool), torch.nan_to_num(v_pool), tables, seq_of, pos, nh, 0.4, None, 0.0)
    for splits in (1, 8, 16, 24):
        got = torch.zeros(1, nh * dv, dtype=torch.bfloat16, device="cuda")
        attn.paged_attention(got, q.cuda(), Cache, Batch(), nh, 0.4, None, splits=splits, sink=0.0)
        _close(got, want, 2e-2, f"splits={splits}")


def test_which_kernels_serve_which_sizes():
    assert ops.prefill_tc_supported(72, 16, 40) and ops.decode_tma_supported(128, 16, 64) and ops.decode_tma_supported(96, 8)
    assert not ops.prefill_tc_supported(136, 16, 64) and not ops.prefill_tc_supported(64, 16, 160) and not ops.decode_tma_supported(32, 16, 32)
    assert not ops.decode_tma_supported(64, 12, 64) and not ops.prefill_tc_supported(64, 48, 128)


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_router_by_softmax_over_all_outputs(dtype, tol):
    for W, E, top in ((48, 6, 2), (64, 13, 3), (50, 7, 7), (128, 40, 12), (256, 16, 1), (32, 1, 1)):
        router, correction = _rand(E, W, seed=1, scale=2.0 / W**0.5), _rand(E, seed=2, scale=0.3)
        for n in (1, 5, 300):
            x = _rand(n, W, seed=10 + n).to(dtype)
            ids_ref, w_ref = torch.zeros(n, top, dtype=torch.int32), torch.zeros(n, top)
            ids_dev, w_dev = ids_ref.cuda(), w_ref.cuda()
            ref.moe_route(ids_ref, w_ref, x, router, correction, 1, 1, 1.5, "softmax")
            ops.moe_route(ids_dev, w_dev, x.cuda(), router.cuda(), correction.cuda(), 1, 1, 1.5, "softmax")
            same = (ids_dev.cpu() == ids_ref).all(1)
            assert same.float().mean() > 0.97, "routing differs on more than near ties"
            _close(w_dev.cpu()[same], w_ref[same], 1e-5, "weights")


@pytest.mark.parametrize("gated", [False, True])
@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("sizes", [(48, 20, 5, 3, 3), (64, 64, 8, 0, 4), (40, 136, 3, 6, 5), (256, 72, 12, 4, 6), (200, 64, 1, 1, 2), (51, 11, 4, 2, 2), (320, 256, 4, 2, 3), (72, 328, 9, 1, 4),
                                   (520, 384, 2, 0, 2)])
def test_experts(sizes, dtype, tol, gated):
    """Experts with and without a gate beside identities, with and without a shared output, for one token, as many as one, two and four
    row tiles of the unsorted kernels hold and one more, and so many that the sort takes several launches; expert counts that leave
    experts without tokens and tokens with identities alone."""
    W, ff, E, identity, top = sizes
    g = torch.Generator().manual_seed(3)
    w_up, w_down = _rand(E, (2 if gated else 1) * ff, W, seed=1, scale=1.0 / W**0.5).to(dtype), _rand(E, W, ff, seed=2, scale=1.0 / ff**0.5).to(dtype)
    act = "silu" if gated else "relu2"
    for n in (1, 3, 16, 17, 33, 64, 65, 700):
        x, shared = _rand(n, W, seed=n).to(dtype), _rand(n, W, seed=n + 1).to(dtype)
        ids = torch.stack([torch.randperm(E + identity, generator=g)[:top] for _ in range(n)]).to(torch.int32)
        if identity >= top:
            ids[0] = torch.arange(E, E + top)  # identities alone
        weights = torch.rand(n, top, generator=g)
        for sh in (shared, None):
            want, got = torch.zeros(n, W, dtype=dtype), torch.full((n, W), 7.0, dtype=dtype, device="cuda")
            ref.moe_experts(want, x, ids, weights, w_up, w_down, act, gated=gated, shared=sh)
            ops.moe_experts(got, x.cuda(), ids.cuda(), weights.cuda(), w_up.cuda(), w_down.cuda(), act, gated=gated, shared=None if sh is None else sh.cuda())
            _close(got, want, tol, f"{n} tokens, shared={sh is not None}")
            if ops.moe_products_supported(W, ff, dtype):  # every form of the products, whatever the step's shape would choose
                for few in (False, True) if n <= ops.MOE_FEW_MAX_TOKENS else (False,):
                    got.fill_(7.0)
                    sums = ops.moe_products(x.cuda(), ids.cuda(), weights.cuda(), w_up.cuda(), w_down.cuda(), act, gated=gated,
                                            shared=None if sh is None else sh.cuda(), few=few)
                    ops.moe_combine(got, sums)
                    _close(got, want, tol, f"{n} tokens, shared={sh is not None}, few={few}")


def test_plain_activations_of_experts():
    x, ids, weights = _rand(6, 64, seed=1), _i32([[0], [1], [0], [1], [0], [1]]), torch.ones(6, 1)
    w_up, w_down = _rand(2, 32, 64, seed=2, scale=0.2), _rand(2, 64, 32, seed=3, scale=0.2)
    for dtype, tol in DTYPES:
        for act in ops.ACTIVATIONS:
            want, got = torch.zeros(6, 64, dtype=dtype), torch.zeros(6, 64, dtype=dtype, device="cuda")
            args = [t.to(dtype) for t in (x, w_up, w_down)]
            ref.moe_experts(want, args[0], ids, weights, args[1], args[2], act, gated=False)
            ops.moe_experts(got, args[0].cuda(), ids.cuda(), weights.cuda(), args[1].cuda(), args[2].cuda(), act, gated=False)
            _close(got, want, tol, act)
    with pytest.raises(ops.KernelError):
        ops.moe_experts(got, args[0].cuda(), ids.cuda(), weights.cuda(), args[1].cuda(), args[2].cuda(), "quick_gelu", gated=False)


@pytest.mark.parametrize("sizes", [(64, 64, 8, 2, 4, 128), (256, 72, 12, 4, 6, 40), (200, 136, 3, 1, 2, 264), (512, 128, 5, 0, 5, 8)])
def test_a_feed_forward_rides_along(sizes):
    """The shared feed-forward in the launches of few tokens' experts, wider and narrower than an expert; the sums added up, and added up,
    normed and added to the stream in one kernel."""
    W, ff, E, identity, top, shared_ff = sizes
    bf = torch.bfloat16
    g = torch.Generator().manual_seed(3)
    w_up, w_down = _rand(E, ff, W, seed=1, scale=1.0 / W**0.5).to(bf), _rand(E, W, ff, seed=2, scale=1.0 / ff**0.5).to(bf)
    s_up, s_down = _rand(shared_ff, W, seed=4, scale=1.0 / W**0.5).to(bf), _rand(W, shared_ff, seed=5, scale=1.0 / shared_ff**0.5).to(bf)
    norm = 1 + 0.2 * _rand(W, seed=6)
    for n in (1, 7, 16, 30, 64):
        x = _rand(n, W, seed=n).to(bf)
        ids = torch.stack([torch.randperm(E + identity, generator=g)[:top] for _ in range(n)]).to(torch.int32)
        weights = torch.rand(n, top, generator=g)
        hidden = torch.relu((x.float() @ s_up.float().t()).to(bf).float()) ** 2
        shared = (hidden.to(bf).float() @ s_down.float().t())
        want = torch.zeros(n, W)
        ref.moe_experts(want, x.float(), ids, weights, w_up.float(), w_down.float(), "relu2", gated=False)
        want += shared
        d = [t.cuda() for t in (x, ids, weights, w_up, w_down)]
        sums = ops.moe_products(*d, "relu2", gated=False, extra=(s_up.cuda(), s_down.cuda(), "relu2"))
        out = torch.empty(n, W, dtype=bf, device="cuda")
        ops.moe_combine(out, sums)
        _close(out, want, 2e-2, f"{n} tokens")
        h = _rand(n, W, seed=9)
        h_dev, y = h.cuda(), torch.empty(n, W, dtype=bf, device="cuda")
        ops.moe_combine_norm_add(h_dev, sums, norm.cuda(), 1e-3, 0.7, y)
        h_want = h + 0.7 * want / torch.sqrt((want * want).mean(-1, keepdim=True) + 1e-3) * norm
        _close(h_dev, h_want, 2e-2, f"{n} tokens, normed and added")
        _close(y, h_want, 2e-2, f"{n} tokens, normed and added, rounded")
        assert (y.float() - h_dev).abs().max() <= 0.01 * h_dev.abs().max()


def test_sums_of_sorted_pairs_are_normed_and_added_too():
    W, ff, E, top, n = 320, 64, 6, 3, 130
    bf = torch.bfloat16
    g = torch.Generator().manual_seed(5)
    x, shared = _rand(n, W, seed=1).to(bf), _rand(n, W, seed=2).to(bf)
    w_up, w_down = _rand(E, ff, W, seed=3, scale=1.0 / W**0.5).to(bf), _rand(E, W, ff, seed=4, scale=1.0 / ff**0.5).to(bf)
    ids = torch.stack([torch.randperm(E + 2, generator=g)[:top] for _ in range(n)]).to(torch.int32)
    weights, norm, h = torch.rand(n, top, generator=g), 1 + 0.2 * _rand(W, seed=6), _rand(n, W, seed=7)
    want = torch.zeros(n, W)
    ref.moe_experts(want, x.float(), ids, weights, w_up.float(), w_down.float(), "relu2", gated=False, shared=shared.float())
    h_dev = h.cuda()
    sums = ops.moe_products(x.cuda(), ids.cuda(), weights.cuda(), w_up.cuda(), w_down.cuda(), "relu2", gated=False, shared=shared.cuda())
    ops.moe_combine_norm_add(h_dev, sums, norm.cuda(), 1e-5, 1.0)
    _close(h_dev, h + want / torch.sqrt((want * want).mean(-1, keepdim=True) + 1e-5) * norm, 2e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("score", ["sigmoid", "softmax", "softmax_chosen"])
def test_routing_does_not_depend_on_how_many_tokens_there_are(dtype, score):
    """The kernel for many tokens adds every sum up in the order of the one for few: the same choices and weights, bit for bit."""
    W, E, top = 264, 21, 5
    x, router, correction = _rand(603, W, seed=1).to(dtype).cuda(), _rand(E, W, seed=2, scale=0.1).cuda(), _rand(E, seed=3, scale=0.2).cuda()
    ids, weights = torch.zeros(603, top, dtype=torch.int32, device="cuda"), torch.zeros(603, top, device="cuda")
    ops.moe_route(ids, weights, x, router, correction, 3, 2, 1.5, score)
    for first in range(0, 603, 201):
        some_ids, some_weights = torch.zeros(201, top, dtype=torch.int32, device="cuda"), torch.zeros(201, top, device="cuda")
        ops.moe_route(some_ids, some_weights, x[first : first + 201].contiguous(), router, correction, 3, 2, 1.5, score)
        assert torch.equal(some_ids, ids[first : first + 201]) and torch.equal(some_weights, weights[first : first + 201])
