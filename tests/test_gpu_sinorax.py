"""Sinorax on the GPU: every new kernel against its plain torch statement, and the engine (both dtypes) against the plain
implementation: whole prompts, decoding token by token, portions down to two tokens, mixed batches on reused pages and slots, long
decoding, greedy generation through the entry point, steps from CUDA graphs, and inputs made so that a far key or the edge of a
window shows in the result."""
from types import SimpleNamespace

import pytest
import torch

from sinorax_cases import (CASES, check_long_decoding, check_mixed, check_slot_reuse, check_whole_and_cut, cuts_of, load_plain, make_folder, plain_logits,
                           prompt, replayer, row_error, run_alone, setup_case)
from torch_kernels import TorchKernels

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
TD = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def K():
    from llm_infrence_engine_b200.csrc import get_kernels

    return get_kernels()


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("sinorax")
    return {(name, dtype): setup_case(tmp, name, dtype) for name in CASES for dtype in DTYPES}


def close(got, want, dtype, what, scale=None, f32=2e-6):
    tol = (f32 if dtype == "float32" else 1.2e-2) * max(1.0, float(want.float().abs().max()) if scale is None else scale)
    err = float((got.float().cpu() - want.float().cpu()).abs().max())
    assert err <= tol, f"{what} ({dtype}): {err:.3g} > {tol:.3g}"


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


# ---------------------------------------------------------------------------------------------------------------------
# kernels

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,H", [(1, 8), (5, 48), (33, 250), (700, 1024), (3, 4100)])
def test_dynamic_tanh_before_and_after_a_sublayer(K, dtype, N, H):
    ref, T = TorchKernels(), TD[dtype]
    x = rnd(N, H, seed=1, scale=2.0)
    pre = (torch.tensor(0.37), 1 + rnd(H, seed=2, scale=0.3), rnd(H, seed=3, scale=0.5))
    post = (torch.tensor(1.9), 1 + rnd(H, seed=4, scale=0.3), rnd(H, seed=5, scale=0.5))
    dpre, dpost = [t.cuda() for t in pre], [t.cuda() for t in post]
    xd = x.clone().cuda()
    close(K.dynamic_tanh(xd, *dpre, T), ref.dynamic_tanh(x, *pre, T), dtype, "dynamic_tanh")
    rows = torch.tensor([N - 1, 0, N - 1], dtype=torch.int32)
    close(K.dynamic_tanh(xd, *dpre, T, rows.cuda()), ref.dynamic_tanh(x, *pre, T, rows), dtype, "dynamic_tanh of rows")
    for y_dtype in (torch.float32, T):
        y = rnd(N, H, seed=6, scale=1.5).to(y_dtype)
        # the addition alone (carried out by flush), then added and passed on in one kernel
        K.post_tanh_add(xd, y.clone().cuda(), *dpost)
        K.flush()
        ref.post_tanh_add(x, y, *post)
        close(xd, x, "float32", "post_tanh_add")
        K.post_tanh_add(xd, y.clone().cuda(), *dpost)
        got = K.dynamic_tanh(xd, *dpre, T)
        ref.post_tanh_add(x, y, *post)
        close(xd, x, "float32", "post_tanh_add inside the next norm")
        close(got, ref.dynamic_tanh(x, *pre, T), dtype, "dynamic_tanh after an addition")
        # chosen rows: the addition is computed for them and not stored
        before = xd.clone()
        K.post_tanh_add(xd, y.clone().cuda(), *dpost)
        got = K.dynamic_tanh(xd, *dpre, T, rows.cuda())
        assert torch.equal(xd, before)
        added = x.clone()
        ref.post_tanh_add(added, y, *post)
        close(got, ref.dynamic_tanh(added, *pre, T, rows), dtype, "dynamic_tanh of rows after an addition")
    # small arguments and large ones: the fast form keeps an absolute error of about 1e-7
    z = torch.cat([torch.linspace(-60, 60, 401), torch.logspace(-8, -1, 111)])[None, :512]
    one, zero, a = torch.ones(512), torch.zeros(512), torch.tensor(1.0)
    zd = torch.zeros(1, 512).cuda()
    K.post_tanh_add(zd, z.to(T).cuda(), a.cuda(), one.cuda(), zero.cuda())
    K.flush()
    assert float((zd.cpu().double() - torch.tanh(z.to(T).double())).abs().max()) < 4e-7
    # a zeroed buffer that a sublayer added into is cleared behind the read, for all rows and for chosen ones
    for rows_ in (None, rows.cuda()):
        buf = K.zeros_like_rows(xd)
        buf += rnd(N, H, seed=7).cuda()
        K.post_tanh_add(xd, buf, *dpost)
        K.dynamic_tanh(xd, *dpre, T, rows_)
        assert float(buf.abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(61, 13, 5), (1, 1, 1), (997, 2000000011, 1999999973)])
def test_bigram_embedding_over_ragged_steps(K, dtype, buckets, mul_prev, mul_cur):
    """Portions, single tokens, a request on a used slot, requests left out of a step, padding rows of a captured step."""
    ref, T, vocab, H = TorchKernels(), TD[dtype], 90, 40
    table, bigram = rnd(vocab, H, seed=1).to(T), rnd(buckets + 1, H, seed=2).to(T)
    last, dlast = torch.full((6, 1), 77, dtype=torch.int32), torch.full((6, 1), 77, dtype=torch.int32).cuda()
    at = {}
    g = torch.Generator().manual_seed(3)
    for step, (slots, lens) in enumerate([([2, 0, 4], [9, 1, 2]), ([0, 2], [1, 5]), ([4, 2, 0], [1, 1, 1]), ([4], [300]), ([2], [2])]):
        if step == 4:
            at[2] = 0          # another request takes the slot over
        starts = [0]
        ids, pos, seq = [], [], []
        for s, n in zip(slots, lens):
            ids += torch.randint(0, vocab, (n,), generator=g).tolist()
            pos += list(range(at.get(s, 0), at.get(s, 0) + n))
            seq += [s] * n
            at[s] = at.get(s, 0) + n
            starts.append(starts[-1] + n)
        R = len(slots)
        if step == 2:          # two padding rows: token 0 at position 0 on the spare slot
            ids, pos, seq, starts, R = ids + [0, 0], pos + [0, 0], seq + [5, 5], starts + [starts[-1] + 1, starts[-1] + 2], R + 2
        t = [torch.tensor(v, dtype=torch.int32) for v in (ids, pos, seq, starts)]
        want = ref.embed_bigram(t[0], table, bigram, buckets, mul_prev, mul_cur, t[1], t[2], t[3], R, last, 1.5)
        d = [v.cuda() for v in t]
        got = K.embed_bigram(d[0], table.cuda(), bigram.cuda(), buckets, mul_prev, mul_cur, d[1], d[2], d[3], R, dlast, 1.5)
        close(got, want, "float32", f"embed_bigram step {step}")
        assert torch.equal(dlast.cpu()[:5], last[:5]), f"last tokens after step {step}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_products_with_a_bias_exact_gelu_and_scaled_cap(K, dtype):
    ref, T = TorchKernels(), TD[dtype]
    for M, N, Kd in ((1, 24, 16), (7, 130, 64), (40, 48, 600), (128, 300, 44), (300, 200, 64), (5, 33, 10)):
        x, w, b = rnd(M, Kd, seed=1).to(T), rnd(N, Kd, seed=2, scale=0.3).to(T), rnd(N, seed=3, scale=3.0).to(T)
        want = ref.linear(x, w, out_dtype=torch.float32, bias=b)
        tol = float(want.abs().max())
        close(K.linear(x.cuda(), w.cuda(), out_dtype=T, bias=b.cuda()), want, dtype, f"linear with a bias {M}x{N}x{Kd}", scale=tol, f32=3e-6)
        close(K.linear(x.cuda(), w.cuda(), out_dtype=torch.float32, bias=b.cuda()), want, "float32", f"linear to float32 {M}x{N}x{Kd}", scale=tol, f32=4e-6)
        y = rnd(M, N, seed=4)
        yd = y.clone().cuda()
        K.linear(x.cuda(), w.cuda(), add_to=yd, bias=b.cuda())
        K.flush()
        close(yd, y + want, dtype, f"linear added with a bias {M}x{N}x{Kd}", scale=tol, f32=4e-6)
        if dtype == "bfloat16" and M <= 128 and Kd % 8 == 0:     # float32 sums for the kernel that follows, split over K
            z = K.linear(x.cuda(), w.cuda(), transient=True, bias=b.cuda())
            close(z, want, "float32", "transient sums with a bias", scale=tol, f32=4e-6)
            z.zero_()
    K.check_device_errors()
    for M, N in ((3, 40), (7, 33), (200, 264), (300, 272), (130, 16), (1100, 1040), (2048, 96)):
        x, w = rnd(M, 64, seed=5).to(T), rnd(N, 64, seed=6, scale=0.3).to(T)
        for act in ("gelu_erf", "gelu_tanh"):
            want = ref.linear_act(x, w, act, T)
            for rows in (1, 1 << 20):      # one kernel with the activation in it, where it takes the sizes; product and activation
                before, K.up_act_min_rows = K.up_act_min_rows, rows
                try:
                    got = K.linear_act(x.cuda(), w.cuda(), act, T)
                finally:
                    K.up_act_min_rows = before
                close(got, want, dtype, f"{act} {M}x{N} (one kernel from {rows} rows)", f32=4e-6)
    if dtype == "bfloat16":   # the fast form of the exact GELU, value by value: a product with the identity
        z = torch.linspace(-12, 12, 256 * 16).to(T).view(256, 16)
        want = ref.linear_act(z.float(), torch.eye(16), "gelu_erf", torch.float32)
        for rows in (z.repeat(4, 1), z, z[:100]):
            got = K.linear_act(rows.contiguous().cuda(), torch.eye(16, dtype=T).cuda(), "gelu_erf", T).float().cpu()
            w_ = want.repeat(4, 1)[:rows.shape[0]]
            assert float(((got - w_).abs() / (w_.abs() * 2 ** -8 + 1e-6)).max()) < 1.0
        K.check_device_errors()
    if dtype == "bfloat16":
        assert K._acc is None or float(K._acc.abs().max()) == 0.0
    x = rnd(9, 77, seed=7, scale=30.0)
    close(K.softcap(x.cuda(), 5.0, 0.3), 5.0 * torch.tanh(0.3 * x / 5.0), "float32", "scaled soft cap")
    close(K.softcap(x.cuda(), None, 0.3), 0.3 * x, "float32", "scale alone")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,dk,dv,dims,inter", [(4, 2, 16, 8, 16, False), (6, 2, 24, 16, 16, True), (3, 1, 64, 64, 64, False), (2, 2, 128, 96, 64, True),
                                                     (3, 3, 64, 40, 32, False), (5, 5, 20, 12, 0, False), (8, 2, 128, 128, 128, False), (1, 1, 10, 6, 2, False)])
def test_heads_and_values_turned_and_stored(K, dtype, nq, nkv, dk, dv, dims, inter):
    ref, T = TorchKernels(), TD[dtype]
    N, page = 19, 8
    slots = (torch.randperm(40, generator=torch.Generator().manual_seed(1))[:N] + 8).to(torch.int32)
    width = (nq + nkv) * dk + nkv * dv
    z = torch.nn.functional.pad(rnd(N, width, seed=2), (0, -width % 8)).to(T)     # (rows are padded by products with rows of zeros)
    pos = torch.arange(N, dtype=torch.int32) * 37
    dc = lambda t: None if t is None else t.cuda()

    def tables(n):
        return ref.rope_tables(pos, 1.0 / (50.0 ** (torch.arange(0, n, 2).float() / n))) if n else (None, None)

    (cos, sin), vt = tables(dims), tables(dv)
    for v_turn in (None, vt):
        pools = [torch.zeros(7, nkv, page, d, dtype=T) for d in (dk, dv)]
        want = ref.qk_norm_rope_store(z, nq, nkv, dk, dv, None, None, 1e-5, cos, sin, dims, inter, slots, *pools, page, v_turn=v_turn)
        dturn = None if v_turn is None else [t.cuda() for t in v_turn]
        ways = ["rows"] + (["sums"] if dtype == "bfloat16" else [])
        for way in ways:
            dpools = [torch.zeros_like(p).cuda() for p in pools]
            zd = z.cuda()
            if way == "sums":      # the float32 sums of a small batch's product, consumed and cleared
                zd = K.linear(torch.eye(z.shape[0], 24, dtype=T).cuda(), torch.nn.functional.pad(z, (0, 0, 0, 5)).T.contiguous().cuda(), transient=True)
            got = K.qk_norm_rope_store(zd, nq, nkv, dk, dv, None, None, 1e-5, dc(cos), dc(sin), dims, inter, slots.cuda(), *dpools, page, v_turn=dturn, out_dtype=T)
            close(got, want, dtype, f"queries ({way})", f32=4e-6)
            close(dpools[0], pools[0], dtype, f"keys in their pages ({way})", f32=4e-6)
            close(dpools[1], pools[1], dtype, f"values in their pages ({way}, turned {v_turn is not None})", f32=4e-6)
            if way == "sums":
                assert float(K._acc.abs().max()) == 0.0
        untouched = [p.clone() for p in dpools]
        K.qk_norm_rope_store(z.cuda(), nq, nkv, dk, dv, None, None, 1e-5, dc(cos), dc(sin), dims, inter, slots.cuda(), *dpools, page, write_kv=False, v_turn=dturn)
        assert torch.equal(dpools[0], untouched[0]) and torch.equal(dpools[1], untouched[1])


def paged(N_ctx, page, nkv, dk, dv, dtype, seed=0):
    """A pool with one request of ``N_ctx`` tokens on shuffled pages; returns pools, block table and the keys/values in order."""
    pages = -(-N_ctx // page)
    perm = (torch.randperm(pages, generator=torch.Generator().manual_seed(seed)) + 1).to(torch.int32)
    k, v = rnd(N_ctx, nkv, dk, seed=seed + 1).to(TD[dtype]), rnd(N_ctx, nkv, dv, seed=seed + 2).to(TD[dtype])
    k_pool, v_pool = torch.zeros(pages + 2, nkv, page, dk, dtype=TD[dtype]), torch.zeros(pages + 2, nkv, page, dv, dtype=TD[dtype])
    for t in range(N_ctx):
        k_pool[perm[t // page], :, t % page] = k[t]
        v_pool[perm[t // page], :, t % page] = v[t]
    table = torch.zeros(3, pages + 1, dtype=torch.int32)
    table[1, :pages] = perm
    return k_pool, v_pool, table, k, v


WAYS = ("generic", "portion", "portion, warp-to-rows kernel", "portion, split-part kernel", "single tokens", "single tokens, split-part kernel", "two equal runs",
        "single tokens, five runs", "single tokens, five runs, split-part kernel")


def run_attention(K, how, q, q_col, common, seq, pos, page, scale, window, ctx_len, **kw):
    """``attention_ext`` by one of the ways its kernels are reached."""
    N = q.shape[0]
    batch, more = None, {}
    if how.startswith("portion") or how == "two equal runs":     # a portion holds neighbouring positions: one per run of them
        starts = [0] + [i for i in range(1, N) if int(pos[i]) != int(pos[i - 1]) + 1] + [N]
        lens = [b - a for a, b in zip(starts, starts[1:])]
        batch = SimpleNamespace(seq_lens=lens, seq_starts_dev=torch.tensor(starts, dtype=torch.int32).cuda(), max_seq_len=max(lens), _tables={})
    if how.startswith("single"):
        batch = SimpleNamespace(seq_lens=[1] * N, seq_starts_dev=torch.arange(N + 1, dtype=torch.int32).cuda(), max_seq_len=1, _tables={})
    if how == "two equal runs":
        more = {"num_splits": 2}
    if "five runs" in how:
        more = {"num_splits": 5}
    K.use_fa_attention_ext = not how.endswith("split-part kernel")
    K.use_plain_attention_for_ext = K.use_tc_attention_ext = not how.endswith("kernel")
    try:
        return K.attention_ext(q.cuda(), q_col, *common, seq.cuda(), pos.cuda(), page, scale, window, ctx_len, batch=batch, **kw, **more)
    finally:
        K.use_fa_attention_ext = K.use_plain_attention_for_ext = K.use_tc_attention_ext = True


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,dk,dv", [(4, 2, 16, 8), (6, 1, 64, 64), (4, 2, 96, 96), (3, 3, 24, 40), (4, 4, 128, 128), (16, 4, 128, 64), (2, 1, 64, 128), (14, 2, 64, 64), (16, 1, 128, 128), (12, 1, 64, 64), (40, 2, 128, 128),
                                          (5, 1, 48, 256), (3, 3, 10, 6)])
def test_attention_sigmoid_penalty_and_turned_values(K, dtype, nq, nkv, dk, dv):
    """Positions spread over a request of 1,300 tokens, as a prompt portion and as single tokens; every kernel that takes the sizes."""
    ctx_len, page = 1300, 16
    k_pool, v_pool, table, _, _ = paged(ctx_len, page, nkv, dk, dv, dtype, 3)
    pos = torch.tensor([0, 1, 5, 15, 16, 17, 100, 199, 200, 201, 1023, 1024, 1025] + list(range(1180, 1213)) + [1299], dtype=torch.int32)
    N = pos.shape[0]
    col = 0 if dk in (64, 128) else 8      # (the kernels of plain attention take rows that begin with the queries)
    q = rnd(N, nq * dk + 8, seed=5, scale=0.5).to(TD[dtype])
    seq = torch.ones(N, dtype=torch.int32)
    pb, r1, r2 = rnd(nq, seed=6) - 2.0, rnd(nq, seed=7).abs() + 0.2, rnd(nq, seed=8).abs() + 0.1
    ang = rnd(N, dv // 2, seed=9, scale=4.0)
    half, near = (torch.cos(ang), torch.sin(ang), False), (torch.cos(ang), torch.sin(ang), True)
    gate = rnd(N, nq * dv + nq, seed=10).to(TD[dtype])
    variants = {
        "sigmoid, penalty, window": (136, dict(sigmoid_bias=pb, log_distance=(r1, r2))),
        "sigmoid alone": (0, dict(sigmoid_bias=pb - 4.0)),
        "sigmoid, window of one": (1, dict(sigmoid_bias=pb, log_distance=(r1, r2))),
        "sigmoid with kept tokens and a gate": (64, dict(sigmoid_bias=pb, keep_first=5, gate=gate, gate_col=nq * dv, gate_per_head=True)),
        "softmax with a penalty": (0, dict(log_distance=(r1, r2))),
        "values turned back": (0, dict(turn=half)),
        "values turned back, neighbours, window": (200, dict(turn=near)),
        "turned back, sink and gate per element": (0, dict(turn=half, sink=rnd(nq, seed=11), gate=gate, gate_col=0)),
        "sigmoid, turned back": (90, dict(sigmoid_bias=pb, turn=half, log_distance=(r1, r2))),
    }
    dev = lambda v: tuple(dev(t) for t in v) if isinstance(v, tuple) else (v.cuda() if torch.is_tensor(v) else v)
    for what, (window, kw) in variants.items():
        want = TorchKernels().attention_ext(q, col, nq, nkv, dk, dv, k_pool, v_pool, table, seq, pos, page, 0.3, window, ctx_len, **kw)
        top = float(want.float().abs().max())
        for how in WAYS:
            got = run_attention(K, how, q, col, (nq, nkv, dk, dv, k_pool.cuda(), v_pool.cuda(), table.cuda()), seq, pos, page, 0.3, window, ctx_len,
                                **{k: dev(v) for k, v in kw.items()})
            # (softmax results are of size 1; sums of sigmoid weights over a thousand keys have a size of their own)
            close(got, want, dtype, f"attention_ext {what} ({how})", scale=8.0 * max(1.0, dk / 64) ** 0.5 * max(1.0, top / 4) if dtype == "float32" else None)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dk,dv", [(32, 16), (64, 64), (96, 96), (128, 64)])
def test_one_key_stands_out_at_the_edges_of_a_window(K, dtype, dk, dv):
    """One key among 1,500 is made to match the query, and the sigmoid's offset shuts all others out: the result is that key's value
    where it is seen and nothing where it is one step outside; at page borders, for a single token and inside a prompt portion."""
    ctx_len, page = 1500, 16
    k_pool, v_pool, table, k, v = paged(ctx_len, page, 1, dk, dv, dtype, 9)
    k_pool = k_pool * 0.02
    unit = torch.zeros(dk)
    unit[5] = 1.0
    pb = torch.tensor([-20.0]).cuda()
    for p, j, window, seen in [(1499, 1499 - 135, 136, True), (1499, 1499 - 136, 136, False), (1499, 1499, 136, True), (136, 0, 136, False), (135, 0, 136, True),
                               (1023, 1008, 16, True), (1023, 1007, 16, False), (1024, 1023, 1, False), (1024, 1024, 1, True), (700, 637, 64, True),
                               (700, 636, 64, False), (255, 0, 256, True), (256, 0, 256, False), (1499, 3, 0, True)]:
        kp = k_pool.clone()
        kp[table[1, j // page], 0, j % page] = (unit * 20.0).to(TD[dtype])
        first = max(0, p - 23)
        q = (unit * 4.0).to(TD[dtype])[None].repeat(p - first + 1, 1)
        pos = torch.arange(first, p + 1, dtype=torch.int32)
        for how in WAYS:
            qq, pp = (q[-1:], pos[-1:]) if how.startswith("single") else (q, pos)
            got = run_attention(K, how, qq, 0, (1, 1, dk, dv, kp.cuda(), v_pool.cuda(), table.cuda()), torch.ones(pp.shape[0], dtype=torch.int32), pp, page, 1.0,
                                window, ctx_len, sigmoid_bias=pb, log_distance=(torch.tensor([0.5]).cuda(), torch.tensor([0.3]).cuda())).float().cpu()[-1]
            want = v[j, 0].float() if seen else torch.zeros(dv)
            d = float((got - want).abs().max())
            assert d < 3e-2, f"key {j} from position {p}, window {window} ({how}): {'seen' if seen else 'not seen'}, off by {d:.3g}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dk,dv", [(32, 16), (64, 64), (96, 96), (128, 128)])
def test_a_far_value_turns_back_by_its_distance(K, dtype, dk, dv):
    """One key owns the softmax; its cached value was turned by its position, and the result is the value turned by the distance."""
    ctx_len, page, base = 1500, 16, 200.0
    k_pool, v_pool, table, k, v = paged(ctx_len, page, 1, dk, dv, dtype, 9)
    f = torch.tensor([base ** (-2.0 * m / dv) for m in range(dv // 2)])
    unit = torch.zeros(dk)
    unit[3] = 1.0
    for p, j in [(1499, 0), (1499, 1498), (1499, 1499), (1023, 15), (1024, 16), (17, 0), (700, 63), (0, 0)]:
        kp, vp = k_pool.clone(), v_pool.clone()
        kp[table[1, j // page], 0, j % page] = (unit * 40.0).to(TD[dtype])
        turned = TorchKernels._turn(v[j:j + 1].float(), torch.cos(j * f)[None], torch.sin(j * f)[None], dv, False)[0, 0]
        vp[table[1, j // page], 0, j % page] = turned.to(TD[dtype])
        first = max(0, p - 23)
        q = (unit * 4.0).to(TD[dtype])[None].repeat(p - first + 1, 1)
        pos = torch.arange(first, p + 1, dtype=torch.int32)
        want = TorchKernels._turn(v[j:j + 1].float(), torch.cos((j - p) * f)[None], torch.sin((j - p) * f)[None], dv, False)[0, 0]
        for how in WAYS:
            qq, pp = (q[-1:], pos[-1:]) if how.startswith("single") else (q, pos)
            a = pp.float()[:, None] * f[None, :]
            got = run_attention(K, how, qq, 0, (1, 1, dk, dv, kp.cuda(), vp.cuda(), table.cuda()), torch.ones(pp.shape[0], dtype=torch.int32), pp, page, 1.0,
                                0, ctx_len, turn=(torch.cos(a).cuda(), torch.sin(a).cuda(), False)).float().cpu()[-1]
            d = float((got - want).abs().max())
            assert d < 4e-2, f"value of {j} read at {p} ({how}): off by {d:.3g}"


def test_refused_combinations(K):
    from llm_infrence_engine_b200.csrc.kernels import KernelError

    k_pool, v_pool, table, _, _ = paged(40, 8, 1, 16, 16, "float32")
    q, seq, pos = rnd(1, 16).cuda(), torch.ones(1, dtype=torch.int32).cuda(), torch.zeros(1, dtype=torch.int32).cuda()
    args = (q, 0, 1, 1, 16, 16, k_pool.cuda(), v_pool.cuda(), table.cuda(), seq, pos, 8, 1.0, 0, 40)
    one = torch.ones(1).cuda()
    for kw in (dict(sigmoid_bias=one, sink=one), dict(sigmoid_bias=torch.ones(2).cuda()), dict(turn=(torch.ones(1, 4).cuda(), torch.ones(1, 4).cuda(), False)),
               dict(talk=torch.eye(1).cuda(), log_distance=(one, one))):
        with pytest.raises(KernelError):
            K.attention_ext(*args, **kw)
    with pytest.raises(KernelError):
        K.linear(q, rnd(4, 16).cuda(), bias=torch.ones(3).cuda())
    with pytest.raises(KernelError):
        K.dynamic_tanh(q, one, torch.ones(15).cuda(), torch.ones(16).cuda(), torch.float32)


# ---------------------------------------------------------------------------------------------------------------------
# the engine

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CASES))
def test_engine_whole_and_cut(cases, name, dtype):
    check_whole_and_cut(cases[(name, dtype)], name, dtype, None, "cuda:0")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CASES))
def test_engine_mixed_batches_on_reused_pages_and_slots(cases, name, dtype):
    check_mixed(cases[(name, dtype)], name, dtype, None, "cuda:0")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CASES))
def test_engine_long_decoding(cases, name, dtype):
    check_long_decoding(cases[(name, dtype)], name, dtype, None, "cuda:0")


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_on_used_slots(cases, dtype):
    for name in ("A", "B", "C"):
        check_slot_reuse(cases[(name, dtype)], name, dtype, None, "cuda:0")


@pytest.mark.parametrize("name", sorted(CASES))
def test_float32_does_not_depend_on_how_the_work_is_cut(cases, name):
    """In float32 the products treat a row by itself, the attention cuts its keys at fixed places and Dynamic Tanh knows no
    neighbours: the same bits whole, in portions, and one by one."""
    folder, cfg, tensors, prompts, want = cases[(name, "float32")]
    rp = replayer(folder, name, "float32", 192)
    p = prompts["e"]
    T = len(p)
    whole = run_alone(rp, "w", p, [(0, T)])
    for n, sizes in enumerate(([7, 2, 33, 1, 16, 3, 2, 64, 5], [T - 30] + [1] * 30, [2])):
        got = run_alone(rp, f"c{n}", p, cuts_of(T, sizes), 1000 * (n + 1))
        assert torch.equal(got, whole), f"{name}: portions of {sizes[:3]} differ by {float((got - whole).abs().max()):.3g}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_sharp_scores_show_a_wrong_key(tmp_path, name, dtype):
    """Query projections several times larger let few keys matter: a key that is lost, read from a wrong page, or seen across the edge
    of a window moves the logits by far more than rounding does. Portions that end on page borders and one off, single tokens
    across the edges."""
    folder = make_folder(tmp_path, name, dtype, sharp=6.0, seed=5)
    cfg, tensors = load_plain(folder)
    p = prompt(cfg["vocab"], 140, 21)
    ref = plain_logits(cfg, tensors, p)
    rp = replayer(folder, name, dtype, 192)
    for n, sizes in enumerate(([140], [8, 8, 1, 7, 9, 15, 16, 17], [100] + [1] * 40, [15] + [1] * 125)):
        got = run_alone(rp, f"s{n}", p, cuts_of(140, sizes), 1000 * n)
        err = row_error(got, ref)
        # (float32 is the sharp detector here; in bfloat16 the sharp scores also magnify the rounding of q and k)
        assert err <= (1e-4 if dtype == "float32" else 0.3), f"sharp {name} {dtype} {sizes[:3]}: {err:.3g}"


def greedy_check(cfg, tensors, prompts, results, dtype):
    for p, r in zip(prompts, results):
        seq = list(p) + r.token_ids
        ref = plain_logits(cfg, tensors, seq)[len(p) - 1:-1]
        if dtype == "float32":
            assert r.token_ids == ref.argmax(-1).tolist()
        else:   # in bfloat16 a near tie may fall the other way: the chosen token must be (nearly) the best one
            chosen = ref.gather(1, torch.tensor(r.token_ids)[:, None])[:, 0]
            assert float((ref.max(-1).values - chosen).max()) <= 0.08 * float(ref.std())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("graphs,pipeline", [(False, False), (True, False), (True, True)])
def test_greedy_generation_through_the_entry_point(cases, dtype, graphs, pipeline):
    """Eager, from graphs, and pipelined (the previous token of a decoded one is then known to the device alone)."""
    from llm_infrence_engine_b200.engine import Engine

    folder, cfg, tensors, prompts, want = cases[("A", dtype)]
    eng = Engine(folder, dtype=dtype, max_len=256, max_seqs=4, block_size=8, num_blocks=70, max_num_batched_tokens=48, cuda_graphs=graphs, pipeline=pipeline)
    if graphs:
        assert eng.runner.graphs.usable, "every part of the model only launches kernels: its decode steps are captured"
    ps = [prompts["c"], prompts["d"], prompts["f"], prompts["b"], prompts["e"][:50]]
    greedy_check(cfg, tensors, ps, eng.generate(ps, max_new_tokens=24), dtype)
    eng.cache.check_invariants()
    assert all(pool.num_free == pool.capacity for pool in eng.cache.pools)


@pytest.mark.parametrize("graphs", [False, True])
def test_a_prompt_in_equal_portions_under_graphs(cases, graphs):
    """A prompt under a small token budget gives step after step of one shape, which is captured while the request is in the middle
    of its prompt: the capture's warm-up must leave the request's last token as it was."""
    from llm_infrence_engine_b200.engine import Engine

    folder, cfg, tensors, prompts, want = cases[("B", "float32")]
    eng = Engine(folder, dtype="float32", max_len=256, max_seqs=2, block_size=16, num_blocks=40, max_num_batched_tokens=16, cuda_graphs=graphs)
    ps = [prompts["a"], prompts["e"]]
    greedy_check(cfg, tensors, ps, [eng.generate([p], max_new_tokens=6)[0] for p in ps], "float32")
    if graphs:
        assert eng.runner.graphs.shape_replays > 3


def test_preemption_starts_from_the_first_token_again(cases):
    """A pool too small for all requests: the youngest is preempted and later recomputed. Same tokens as with room for all."""
    from llm_infrence_engine_b200.engine import Engine

    folder, cfg, tensors, prompts, want = cases[("B", "float32")]
    ps = [prompts["b"], prompts["c"], prompts["a"][:60], prompts["e"][:70]]
    big = Engine(folder, dtype="float32", max_len=160, max_seqs=4, block_size=16, num_blocks=60, max_num_batched_tokens=64)
    want_tokens = [r.token_ids for r in big.generate(ps, max_new_tokens=40)]
    small = Engine(folder, dtype="float32", max_len=160, max_seqs=4, block_size=16, num_blocks=19, max_num_batched_tokens=64)
    got = [r.token_ids for r in small.generate(ps, max_new_tokens=40)]
    assert small.preemptions > 0 and got == want_tokens
    small.cache.check_invariants()


def test_random_weights_and_the_command_line(tmp_path):
    import json
    import subprocess
    import sys
    from pathlib import Path

    root = Path(__file__).resolve().parent.parent
    (tmp_path / "cfg.json").write_text(json.dumps(CASES["D"][0]))
    out = subprocess.run([sys.executable, "-m", "llm_infrence_engine_b200", "--model", str(tmp_path / "m"), "--random-weights", str(tmp_path / "cfg.json"),
                          "--dtype", "float32", "--prompt-ids", "1 2 3 4 5", "--max-new-tokens", "6", "--max-len", "64", "--max-seqs", "2"],
                         cwd=root, capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    tokens = json.loads(out.stdout.strip().splitlines()[0])["token_ids"]
    cfg, tensors = load_plain(tmp_path / "m")
    seq = [1, 2, 3, 4, 5]
    for t in tokens:
        assert t == int(plain_logits(cfg, tensors, seq)[-1].argmax())
        seq.append(t)
