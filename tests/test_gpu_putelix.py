"""Putelix on the GPU: every new kernel against its plain torch statement, and the engine (both dtypes) against the plain
implementation: whole prompts, decoding token by token, portions down to two tokens, mixed batches on reused pages and slots, long
decoding, greedy generation through the entry point, steps from CUDA graphs, and inputs made so that a far key, the edge of a chunk or
a lost state shows in the result."""
from types import SimpleNamespace

import pytest
import torch

from putelix_cases import (CASES, check_long_decoding, check_mixed, check_slot_reuse, check_whole_and_cut, cuts_of, judge, load_plain, make_folder, plain_logits,
                           prompt, replayer, run_alone, setup_case, tapped_alone)
from test_gpu_sinorax import WAYS, paged, run_attention
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
    tmp = tmp_path_factory.mktemp("putelix")
    return {(name, dtype): setup_case(tmp, name, dtype) for name in CASES for dtype in DTYPES}


def close(got, want, dtype, what, scale=None, f32=2e-6):
    tol = (f32 if dtype == "float32" else 1.2e-2) * max(1.0, float(want.float().abs().max()) if scale is None else scale)
    err = float((got.float().cpu() - want.float().cpu()).abs().max())
    assert err <= tol, f"{what} ({dtype}): {err:.3g} > {tol:.3g}"


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def ragged(lens, slots):
    """The description of a step whose requests bring ``lens`` rows and own the state rows ``slots``."""
    starts = [0]
    for n in lens:
        starts.append(starts[-1] + n)
    host = SimpleNamespace(seq_starts_dev=torch.tensor(starts, dtype=torch.int32), seq_slots=torch.tensor(slots, dtype=torch.int32),
                           num_seqs=len(lens), max_seq_len=max(lens), seq_lens=list(lens), _tables={})
    dev = SimpleNamespace(**{**host.__dict__, "seq_starts_dev": host.seq_starts_dev.cuda(), "seq_slots": host.seq_slots.cuda(), "_tables": {}})
    return host, dev


# ---------------------------------------------------------------------------------------------------------------------
# kernels

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [8, 44, 250, 1024])
def test_embedding_with_positions(K, dtype, H):
    T = TD[dtype]
    table, pos_table = rnd(30, H, seed=1).to(T), rnd(17, H, seed=2).to(T)
    ids, pos = torch.tensor([3, 0, 29, 3, 3], dtype=torch.int32), torch.tensor([0, 16, 5, 1, 0], dtype=torch.int32)
    for scale in (1.0, 2.5):
        got = K.embed_positions(ids.cuda(), table.cuda(), pos.cuda(), pos_table.cuda(), scale)
        close(got, TorchKernels().embed_positions(ids, table, pos, pos_table, scale), "float32", "embedding with positions", f32=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,H", [(1, 8), (5, 48), (33, 250), (200, 1024), (3, 4100), (2, 9000), (2, 4099)])
def test_closing_norm_join_of_two_and_rows_of_the_stream(K, dtype, N, H):
    ref, T = TorchKernels(), TD[dtype]
    w, wa, wb, wf = (1 + rnd(H, seed=s, scale=0.2) for s in (2, 3, 4, 5))
    rows = torch.tensor([N - 1, 0], dtype=torch.int32)
    dw, dwa, dwb, dwf = (t.cuda() for t in (w, wa, wb, wf))
    types = [torch.float32] if dtype == "float32" else [torch.float32, torch.bfloat16]
    x = rnd(N, H, seed=1)
    xd = x.cuda()
    close(K.stream_rows(xd, T), x.to(T), dtype, "rows as they are")
    assert K.stream_rows(xd, torch.float32) is xd
    for ta in types:
        for tb in [None] + types:
            a = (rnd(N, H, seed=6, scale=3.0) + 0.5).to(ta)
            b = None if tb is None else rnd(N, H, seed=7, scale=0.2).to(tb)

            def start():
                """The result (or the pair of results) on its way into the stream; the oracle's copy of the result."""
                y = K.zeros_like_rows(xd)
                if b is None:
                    r = a.float()
                    if ta == torch.float32:
                        y += a.cuda()
                        K.flush()
                    else:
                        K._pending_add = (y, a.cuda())    # (a library product that still waits)
                else:
                    r = torch.zeros(N, H)
                    ref.dual_rmsnorm_mix(a, b, wa, wb, 1e-5, 0.5, r)
                    K.dual_rmsnorm_mix(a.cuda(), b.cuda(), dwa, dwb, 1e-5, 0.5, y)
                K.post_rms_add(xd, y, dw, 1e-5)
                return r, y

            what = f"{ta} and {tb}"
            r, y = start()
            ref.post_rms_add(x, r, w, 1e-5)
            K.flush()                                       # alone
            close(xd, x, "float32", f"closing norm ({what})", f32=4e-6)
            assert float(y.abs().max()) == 0.0
            r, y = start()
            ref.post_rms_add(x, r, w, 1e-5)
            got = K.stream_rows(xd, T)                      # with the rows of the next sublayer
            close(xd, x, "float32", f"closing norm ({what}) with the next rows", f32=4e-6)
            close(got, x.to(T), dtype, f"the next rows ({what})", f32=4e-6)
            before = xd.clone()
            r, y = start()
            got = K.rmsnorm_rows(xd, None, dwf, 1e-5, rows.cuda(), T)     # with the last norm, of chosen rows
            after = x.clone()
            ref.post_rms_add(after, r, w, 1e-5)
            close(got, ref.rmsnorm_rows(after, None, wf, 1e-5, rows, T), dtype, f"the last norm ({what})", f32=4e-6)
            assert torch.equal(xd, before) and float(y.abs().max()) == 0.0
    # a pair that somebody else reads is carried out first, and a pair into a tensor that holds something is added
    y = K.zeros_like_rows(xd)
    a, b = rnd(N, H, seed=8), rnd(N, H, seed=9)
    K.dual_rmsnorm_mix(a.cuda(), b.cuda(), dwa, dwb, 1e-5, 0.5, y)
    K.dual_rmsnorm_mix(a.cuda(), b.cuda(), dwa, dwb, 1e-5, 0.5, K.take_result(y))
    r = torch.zeros(N, H)
    ref.dual_rmsnorm_mix(a, b, wa, wb, 1e-5, 1.0, r)
    close(y, r, "float32", "two pairs", f32=4e-6)
    y.zero_()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,dk,dv,gates", [(4, 2, 16, 16, 4), (6, 2, 40, 40, 6), (3, 1, 10, 10, 3), (8, 2, 64, 64, 0), (2, 2, 22, 6, 2), (16, 4, 128, 128, 16), (1, 1, 32, 40, 1)])
def test_rows_normed_and_stored(K, dtype, nq, nkv, dk, dv, gates):
    ref, T = TorchKernels(), TD[dtype]
    N, page = 19, 8
    slots = (torch.randperm(40, generator=torch.Generator().manual_seed(1))[:N] + 8).to(torch.int32)
    wq, wk = 1 + rnd(nq * dk, seed=2, scale=0.3), 1 + rnd(nkv * dk, seed=3, scale=0.3)
    for shared in (True, False):
        if shared and dk != dv:
            continue
        width = (nq + nkv) * dk + (0 if shared else nkv * dv) + gates
        z = torch.nn.functional.pad(rnd(N, width, seed=4, scale=2.0), (0, -width % 8)).to(T)
        pools = [torch.zeros(7, nkv, page, d, dtype=T) for d in (dk, dv)]
        scale = torch.zeros(7, page) if shared else None
        want = ref.qk_rows_norm_store(z, nq, nkv, dk, dv, wq, wk, 1e-5, slots, pools[0], None if shared else pools[1], scale, page, gate_cols=gates)
        for way in ["rows"] + (["sums"] if dtype == "bfloat16" else []):
            dpools = [torch.zeros_like(p).cuda() for p in pools]
            dscale = torch.zeros(7, page).cuda() if shared else None
            zd = z.cuda()
            if way == "sums":      # the float32 sums of a small batch's product, consumed and cleared
                zd = K.linear(torch.eye(N, 24, dtype=T).cuda(), torch.nn.functional.pad(z, (0, 0, 0, 5)).T.contiguous().cuda(), transient=True)
            args = (nq, nkv, dk, dv, wq.cuda(), wk.cuda(), 1e-5, slots.cuda(), dpools[0], None if shared else dpools[1], dscale, page)
            got = K.qk_rows_norm_store(zd, *args, gate_cols=gates, out_dtype=T)
            assert got.shape == want.shape and got.shape[1] % 8 == 0
            close(got, want, dtype, f"queries and gate ({way})", f32=4e-6)
            close(dpools[0], pools[0], dtype, f"keys in their pages ({way}, values of their own {not shared})", f32=4e-6)
            if shared:
                close(dscale, scale, "float32", "a number per token", f32=2e-6 if dtype == "float32" or way == "sums" else 4e-6)
            else:
                close(dpools[1], pools[1], dtype, "values in their pages", f32=4e-6)
            if way == "sums":
                assert float(K._acc.abs().max()) == 0.0
        untouched = [p.clone() for p in dpools]
        K.qk_rows_norm_store(z.cuda(), *args, gate_cols=gates, write_kv=False)
        assert all(torch.equal(a, b) for a, b in zip(dpools, untouched))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,d", [(4, 2, 16), (6, 1, 64), (6, 2, 48), (4, 2, 96), (4, 4, 128), (16, 4, 128), (14, 2, 64), (12, 1, 64), (40, 1, 128), (3, 3, 10), (5, 1, 256)])
def test_attention_on_shared_rows(K, dtype, nq, nkv, d):
    """Keys that are values too, with a number per token: positions spread over a request of 1,300 tokens, as a prompt portion and as
    single tokens; every kernel that takes the sizes."""
    ctx_len, page = 1300, 16
    k_pool, _, table, _, _ = paged(ctx_len, page, nkv, d, d, dtype, 3)
    scalar = rnd(k_pool.shape[0], page, seed=4).abs() + 0.2
    pos = torch.tensor([0, 1, 5, 15, 16, 17, 100, 199, 200, 201, 1023, 1024, 1025] + list(range(1180, 1213)) + [1299], dtype=torch.int32)
    N = pos.shape[0]
    col = 0 if d in (64, 128) else 8
    q = rnd(N, nq * d + 8, seed=5, scale=0.4).to(TD[dtype])
    seq = torch.ones(N, dtype=torch.int32)
    gate = rnd(N, nq * d + nq, seed=10).to(TD[dtype])
    rel = rnd(9, nq, seed=6)
    rows = torch.tensor([min(8, n // 20) for n in range(170)], dtype=torch.int32)
    variants = {
        "alone": dict(),
        "chunk, cap, bias and gate": dict(chunk=64, softcap=4.0, rel=rel, rel_rows=rows, gate=gate, gate_col=nq * d, gate_per_head=True),
        "chunk longer than the request": dict(chunk=5000, softcap=2.0, rel=rel, rel_rows=rows),
        "chunk of one": dict(chunk=1, rel=rel, rel_rows=rows),
        "cap, sink and gate per element": dict(softcap=3.0, sink=rnd(nq, seed=11), gate=gate, gate_col=0),
        "penalty by distance": dict(log_distance=(rnd(nq, seed=7).abs(), rnd(nq, seed=8).abs()), chunk=300),
        "sigmoid weights": dict(sigmoid_bias=rnd(nq, seed=9) - 4.0),
    }
    dev = lambda v: tuple(dev(t) for t in v) if isinstance(v, tuple) else (v.cuda() if torch.is_tensor(v) else v)
    for what, kw in variants.items():
        want = TorchKernels().attention_ext(q, col, nq, nkv, d, d, k_pool, None, table, seq, pos, page, 0.3, 0, ctx_len, key_scale=scalar, **kw)
        top = float(want.float().abs().max())
        for how in WAYS:
            got = run_attention(K, how, q, col, (nq, nkv, d, d, k_pool.cuda(), None, table.cuda()), seq, pos, page, 0.3, 0, ctx_len, key_scale=scalar.cuda(),
                                **{k: dev(v) for k, v in kw.items()})
            close(got, want, dtype, f"attention_ext {what} ({how})", scale=8.0 * max(1.0, d / 64) ** 0.5 * max(1.0, top / 4) if dtype == "float32" else None)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [32, 64, 96, 128])
def test_one_key_stands_out_at_the_edges_of_a_chunk(K, dtype, d):
    """One key among 1,500 is made to match the query and owns the softmax where it is seen; its number per token makes the difference, the
    row itself is no larger than its neighbours' in that direction. At page borders, for a single token and inside a prompt portion."""
    ctx_len, page = 1500, 16
    k_pool, _, table, k, _ = paged(ctx_len, page, 1, d, d, dtype, 9)
    k_pool[..., 5] = 1.0                   # every key has the query's direction ...
    for p, j, chunk, seen in [(1499, 1472, 64, True), (1499, 1471, 64, False), (1499, 1499, 64, True), (128, 127, 128, False), (128, 128, 128, True), (127, 0, 128, True),
                              (1023, 1008, 16, True), (1023, 1007, 16, False), (1024, 1023, 1, False), (1024, 1024, 1, True), (700, 600, 200, True), (700, 599, 200, False),
                              (719, 680, 40, True), (720, 719, 40, False), (1499, 3, 0, True)]:
        scalar = torch.full((k_pool.shape[0], page), 0.01)
        scalar[table[1, j // page], j % page] = 4.0      # ... and one has the number that lets it win
        first = max(0, p - 23)
        q = torch.zeros(p - first + 1, d)
        q[:, 5] = 6.0
        pos = torch.arange(first, p + 1, dtype=torch.int32)
        for how in WAYS:
            qq, pp = (q[-1:], pos[-1:]) if how.startswith("single") else (q, pos)
            got = run_attention(K, how, qq.to(TD[dtype]), 0, (1, 1, d, d, k_pool.cuda(), None, table.cuda()), torch.ones(pp.shape[0], dtype=torch.int32), pp, page, 1.0,
                                0, ctx_len, chunk=chunk, key_scale=scalar.cuda()).float().cpu()[-1]
            value = k_pool[table[1, j // page], 0, j % page].float()
            off = float((got - value).abs().max())
            assert (off < 4e-2) if seen else (off > 0.3), f"key {j} from position {p}, chunk {chunk} ({how}): off by {off:.3g}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,DV", [(1, 8, 8), (3, 64, 32), (2, 128, 128), (4, 16, 40), (1, 256, 24), (2, 14, 6), (5, 96, 64), (2, 104, 8), (1, 200, 16), (2, 20, 7), (1, 1, 1)])
def test_linear_attention(K, dtype, H, D, DV):
    """Requests of unequal length in one step, single tokens among them, on shuffled state rows; then a second step from the states that
    the first one left. The scan and, in bfloat16, the form on the tensor cores."""
    ref, T = TorchKernels(), TD[dtype]
    pad = lambda n: n + -n % 8
    qc, kc, vc = 0, pad(H * D), 2 * pad(H * D)
    width = vc + 2 * pad(H * DV)
    decay = torch.tensor([0.999, 0.5, 0.0, 1.0, 0.93][:H])
    forms = [False] + ([True] if dtype == "bfloat16" and K.lib.llmie_linear_attention_mma_fits(D, DV) else [])
    for lens, slots in (([1, 1, 1], [2, 0, 3]), ([70, 1, 64, 3], [1, 3, 0, 2]), ([130], [2]), ([63, 65, 129, 2], [3, 2, 1, 0])):
        host, dev = ragged(lens, slots)
        for activated, step_kernel in [(f, True) for f in forms] + ([(False, False)] if dtype == "bfloat16" and max(lens) == 1 else []):
            K.use_linear_attention_step = step_kernel
            state = rnd(5, H, DV, D, seed=1, scale=0.5)
            sd = state.cuda()
            for step in range(2):
                z = rnd(sum(lens), width, seed=2 + step).to(T)
                want = ref.linear_attention(z, qc, kc, vc, H, D, DV, decay, state, host, activated=activated)
                got = K.linear_attention(z.cuda(), qc, kc, vc, H, D, DV, decay.cuda(), sd, dev, activated=activated)
                size = float(want.abs().max())
                # (the tensor-core form keeps 16 bits of the numbers it multiplies)
                close(got, want, "float32", f"{lens} step {step} activated {activated}", scale=size, f32=3e-5 if activated else 4e-6)
                close(sd, state, "float32", f"states after {lens} step {step}", scale=float(state.abs().max()), f32=3e-5 if activated else 4e-6)
            assert torch.equal(sd[4].cpu(), state[4])
            K.use_linear_attention_step = True


def test_linear_attention_remembers_the_first_token(K):
    """A decay of 1: the first token's value comes back unweakened a thousand tokens later, whatever lies between, in one portion, cut, and
    decoded on; a decay of 0: only the token itself."""
    H, D, DV, N = 2, 64, 32, 1000
    decay = torch.tensor([1.0, 0.0]).cuda()
    z = torch.zeros(N, 2 * H * D + H * DV)
    q, k, v = z[:, :H * D].view(N, H, D), z[:, H * D:2 * H * D].view(N, H, D), z[:, 2 * H * D:].view(N, H, DV)
    k[0, :, 3] = 1.0
    v[0] = rnd(H, DV, seed=1)
    q[0, :, 3] = q[-1, :, 3] = 2.0
    k[1:, :, 7] = 1.0
    v[1:] = rnd(N - 1, H, DV, seed=2)
    zb = z.to(torch.bfloat16).cuda()
    first = 2 * zb[0, 2 * H * D:].float().view(H, DV).cpu()
    for cuts in ([N], [64, 64, 1, 2, 63, 65, 300, N - 559], [N - 1, 1], [1, N - 1]):
        state = torch.zeros(2, H, DV, D).cuda()
        outs, at = [], 0
        for n in cuts:
            _, dev = ragged([n], [1])
            outs.append(K.linear_attention(zb[at:at + n].contiguous(), 0, H * D, 2 * H * D, H, D, DV, decay, state, dev, activated=True))
            at += n
        o = torch.cat(outs).view(N, H, DV).cpu()
        assert float((o[0] - first).abs().max()) < 1e-5
        assert float((o[-1, 0] - first[0]).abs().max()) < 1e-4 and float(o[-1, 1].abs().max()) < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("act", ["relu2", "silu"])
def test_products_with_squared_relu_and_silu(K, dtype, act):
    ref, T = TorchKernels(), TD[dtype]
    for M, N_, K_ in ((1, 72, 48), (9, 50, 44), (128, 96, 64), (300, 112, 64), (600, 256, 128), (1100, 160, 72)):
        x, w = rnd(M, K_, seed=1).to(T), rnd(N_, K_, seed=2, scale=K_ ** -0.5).to(T)
        got = K.linear_act(x.cuda(), w.cuda(), act, T)
        close(got, ref.linear_act(x, w, act, T), dtype, f"{act} {M}x{N_}", f32=4e-6)
    if dtype == "bfloat16":
        assert K._acc is None or float(K._acc.abs().max()) == 0.0
        K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
def test_router_with_bias_and_gates(K, dtype):
    ref, T = TorchKernels(), TD[dtype]
    for N, W, E, top, gates in ((1, 44, 4, 1, 1), (7, 64, 6, 6, 0), (33, 256, 40, 8, 2), (5, 128, 129, 40, 1), (300, 256, 32, 4, 1), (200, 64, 300, 3, 0)):
        h, w, bias = rnd(N, W, seed=1).to(T), rnd(E + gates, W, seed=2, scale=2 * W ** -0.5).to(T), rnd(E, seed=3)
        for scoring in ("top_softmax", "softmax", "sigmoid"):
            ids, wts, g = K.moe_router(h.cuda(), w.cuda(), None, top, scoring=scoring, bias=bias.cuda(), gates=gates)
            ids2, wts2, g2 = ref.moe_router(h, w, None, top, scoring=scoring, bias=bias, gates=gates)
            logits = h.float() @ w.float().T
            z = logits[:, :E] + bias
            chosen = z.gather(1, ids.cpu().long())
            assert all(len(set(row)) == top for row in ids.cpu().tolist())
            # (of nearly equal logits either may be taken: the chosen ones are as large as the oracle's)
            assert float((chosen - z.gather(1, ids2.long())).abs().max()) < 2e-4, (N, E, scoring)
            close(wts.sort(-1).values, wts2.sort(-1).values, "float32", f"weights {scoring} {N}x{E}", f32=2e-4)
            if gates:
                close(g, g2, "float32", "gates", f32=2e-4)
    big = torch.tensor([[300.0, -300.0, 299.0, 0.0]])
    ids, wts, g = K.moe_route(big.cuda(), None, 2, scoring="top_softmax", gates=1)
    assert ids.tolist() == [[0, 2]] and float(g) == 0.5
    close(wts, torch.softmax(torch.tensor([[300.0, 299.0]]), -1), "float32", "far logits")


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_unit_with_a_scale_per_row(K, dtype):
    ref, T = TorchKernels(), TD[dtype]
    for M, I, W in ((1, 28, 44), (9, 48, 64), (200, 64, 64), (300, 96, 72), (1100, 128, 64)):
        x, w = rnd(M, W, seed=1).to(T), rnd(2 * I, W, seed=2, scale=W ** -0.5).to(T)
        s = torch.rand(M, 1, generator=torch.Generator().manual_seed(3))
        got = K.gate_up_act(x.cuda(), w.cuda(), T, row_scale=s.cuda())
        close(got, ref.gate_up_act(x, w, T, row_scale=s), dtype, f"scaled unit {M}x{I}", f32=4e-6)
        assert torch.equal(K.gate_up_act(x.cuda(), w.cuda(), T, row_scale=torch.zeros(M).cuda()), torch.zeros(M, I, dtype=T).cuda())
    K.check_device_errors()


def test_refused_combinations(K):
    from llm_infrence_engine_b200.csrc.kernels import KernelError

    k_pool, _, table, _, _ = paged(40, 8, 1, 16, 16, "float32")
    q, seq, pos = rnd(1, 16).cuda(), torch.ones(1, dtype=torch.int32).cuda(), torch.zeros(1, dtype=torch.int32).cuda()
    args = (q, 0, 1, 1, 16, 16, k_pool.cuda(), None, table.cuda(), seq, pos, 8, 1.0, 0, 40)
    for kw in (dict(key_scale=torch.ones(3, 8).cuda()), dict(key_scale=torch.ones(k_pool.shape[0], 8).cuda(), talk=torch.eye(1).cuda())):
        with pytest.raises(KernelError):
            K.attention_ext(*args, **kw)
    with pytest.raises(KernelError):
        K.gate_up_act(q, rnd(8, 16).cuda(), row_scale=torch.ones(2).cuda())
    with pytest.raises(KernelError):
        K.moe_router(q, rnd(5, 16).cuda(), None, 2, scoring="top_softmax", bias=torch.ones(5).cuda(), gates=1)
    with pytest.raises(KernelError):
        K.linear_attention(q, 0, 0, 0, 1, 16, 16, torch.ones(2).cuda(), torch.zeros(2, 1, 16, 16).cuda(), ragged([1], [0])[1])


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
    """In float32 the products treat a row by itself, the attention cuts its keys at fixed places and the recurrence walks its tokens in
    order: the same bits whole, in portions, and one by one."""
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
    """Queries several times larger let few keys matter: a key that is lost, read from a wrong page, or seen across the edge of a chunk
    moves the logits by far more than rounding does. Portions that end on page borders and one off, single tokens across the edges."""
    folder = make_folder(tmp_path, name, dtype, sharp=6.0, seed=5)
    cfg, tensors = load_plain(folder)
    p = prompt(cfg["vocab"], 140, 21)
    ref = plain_logits(cfg, tensors, p)
    rp = replayer(folder, name, dtype, 192)
    for n, sizes in enumerate(([140], [8, 8, 1, 7, 9, 15, 16, 17], [100] + [1] * 40, [15] + [1] * 125)):
        got, choices = tapped_alone(rp, cfg, f"s{n}", p, cuts_of(140, sizes), 1000 * n)
        # (float32 is the sharp detector here; in bfloat16 the sharp scores also magnify the rounding of q and k)
        judge(got, (folder, cfg, tensors), p, choices, dtype, f"sharp {name} {dtype} {sizes[:3]}", ref, 1e-4 if dtype == "float32" else 0.3)


def greedy_check(cfg, tensors, prompts, results, dtype):
    for p, r in zip(prompts, results):
        seq = list(p) + r.token_ids
        ref = plain_logits(cfg, tensors, seq)[len(p) - 1:-1]
        if dtype == "float32":
            assert r.token_ids == ref.argmax(-1).tolist()
        else:   # in bfloat16 a near tie may fall the other way: the chosen token must be (nearly) the best one
            chosen = ref.gather(1, torch.tensor(r.token_ids)[:, None])[:, 0]
            assert float((ref.max(-1).values - chosen).max()) <= 0.1 * float(ref.std())


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


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("graphs", [False, True])
def test_a_prompt_in_equal_portions_under_graphs(cases, graphs, dtype):
    """A prompt under a small token budget gives step after step of one shape, which is captured while the request is in the middle
    of its prompt: the capture's warm-up must leave the request's state as it was."""
    from llm_infrence_engine_b200.engine import Engine

    folder, cfg, tensors, prompts, want = cases[("B", dtype)]
    eng = Engine(folder, dtype=dtype, max_len=256, max_seqs=2, block_size=16, num_blocks=40, max_num_batched_tokens=16 if dtype == "float32" else 32, cuda_graphs=graphs)
    ps = [prompts["a"], prompts["e"]]
    greedy_check(cfg, tensors, ps, [eng.generate([p], max_new_tokens=6)[0] for p in ps], dtype)
    if graphs:
        assert eng.runner.graphs.shape_replays > 1


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
