"""Fuvozen on the GPU against the plain float64 oracle (tests/fuvozen_oracle.py): each mechanism's kernel alone, then whole models through
the engine's step function — prompt pass vs token-by-token decoding, portions down to two tokens, cache rows and every carried state
reused by a second request, keys far away and at the borders of the window and of the kernels' key groups, the first tokens, sizes that
are odd, 1 or equal where the usual ones differ, long decoding with and without graph replay, and greedy generation through the engine's
entry point."""
import ctypes as C

import numpy as np
import pytest
import torch

import fuvozen_oracle as O
from fuvozen_util import device_tensors
from zelunex_util import rel_rms, write_model_dir

from ntransformer_b200._lib import lib
from ntransformer_b200.dtypes import DType
from ntransformer_b200.engine import Engine, Model

pytestmark = pytest.mark.gpu

TORCH_DT = {DType.F32: torch.float32, DType.BF16: torch.bfloat16}


def dev(a, dt=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).cuda().to(dt).contiguous()


def stream():
    return torch.cuda.current_stream().cuda_stream


def host(t):
    return t.double().cpu().numpy()


_KEPT = []


def dp(a, dt=torch.float32):
    """Device pointer of a fresh copy of `a`; the copy lives until the test ends (the launches are asynchronous)."""
    t = dev(a, dt)
    _KEPT.append(t)
    return t.data_ptr()


@pytest.fixture(autouse=True)
def _release_kept():
    yield
    torch.cuda.synchronize()
    _KEPT.clear()


def ptrs(ts):
    return (C.c_void_p * len(ts))(*[t.data_ptr() if isinstance(t, torch.Tensor) else t for t in ts])


def ints(v):
    return (C.c_int * len(v))(*v)


def joined(split, rows, cols):
    """hi + lo of a BF16 split workspace, the live rows."""
    mp = (rows + 127) // 128 * 128
    w = split.view(torch.bfloat16).reshape(2, mp, cols)
    return host(w[0, :rows]) + host(w[1, :rows])


def split_buffer(rows, cols):
    return torch.zeros(2 * ((rows + 127) // 128 * 128) * cols, device="cuda", dtype=torch.bfloat16)


# ---------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(7, 3, 5), (1, 1, 1), (1021, 999983, 2654435761)])
def test_pair_embedding_carries_the_previous_token(dt, buckets, mul_prev, mul_cur):
    rng = np.random.default_rng(buckets)
    T, V, W = 23, 50, 19
    E, B = O.bf16_grid(rng.standard_normal((V, W))), O.bf16_grid(rng.standard_normal((buckets + 1, W)))
    toks = rng.integers(0, V, T)
    ref = E[toks] + B[O.bigram_rows(toks, buckets, mul_prev, mul_cur)]
    td = torch.from_numpy(toks.astype(np.int32)).cuda()
    e, b = dev(E, TORCH_DT[dt]), dev(B, TORCH_DT[dt])
    for sizes in ([T], [1] * T, [2, 1, 20]):
        pos = 0
        for n in sizes:
            x0, x1 = torch.empty(n, W, device="cuda"), torch.empty(n, W, device="cuda")
            prev = td[max(pos - 1, 0):].clone() if pos else torch.full((1,), 49, device="cuda", dtype=torch.int32)      # stale at position 0
            cur = td[pos:pos + n].clone()
            lib().nt_b200_embed_pair_rows(x0.data_ptr(), x1.data_ptr(), e.data_ptr(), b.data_ptr(), int(dt), cur.data_ptr(), prev.data_ptr(), n, W, buckets, mul_prev,
                                          mul_cur, pos, stream())
            np.testing.assert_allclose(host(x0), ref[pos:pos + n], rtol=1e-6, atol=1e-6)
            np.testing.assert_array_equal(host(x0), host(x1))
            pos += n


@pytest.mark.parametrize("width,groups,n", [(36, 3, 1), (36, 1, 4), (40, 5, 2), (7, 7, 3), (1, 1, 2), (6000, 1, 3), (6000, 3, 2), (8192, 4, 6), (5003, 1, 2)])
def test_depth_average_and_grouped_norm(width, groups, n):
    rng = np.random.default_rng(width + n)
    T, eps = 5, 1e-3
    X = rng.standard_normal((n, T, width)) * np.exp(rng.uniform(-2, 2, (1, 1, width)))        # groups of unequal size: a norm over the whole row would show
    c, g = rng.standard_normal(n), 1 + 0.3 * rng.standard_normal(width)
    for coef in (c, None):
        x_ref = O.depth_average(list(X), c) if coef is not None else X[-1]
        h_ref = O.norm_groups(x_ref, g, groups, eps)
        xs = dev(X)
        xo, ho = torch.empty(T, width, device="cuda"), torch.empty(T, width, device="cuda")
        sp = split_buffer(T, width)
        lib().nt_b200_depth_norm_rows(xs.data_ptr(), T * width, n, dp(coef) if coef is not None else None, xo.data_ptr(), ho.data_ptr(), sp.data_ptr(), dp(g), eps, T, width,
                                      groups, 0, None, None, None, 0, stream())
        np.testing.assert_allclose(host(xo), x_ref, rtol=2e-5, atol=2e-5 * np.abs(x_ref).max())
        np.testing.assert_allclose(host(ho), h_ref, rtol=2e-5, atol=3e-5)
        np.testing.assert_allclose(joined(sp, T, width), h_ref, rtol=1e-4, atol=1e-4)
        xo.zero_()
        lib().nt_b200_depth_norm_rows(xs.data_ptr(), T * width, n, dp(coef) if coef is not None else None, xo.data_ptr(), None, None, None, eps, T, width, groups, 0, None,
                                      None, None, 0, stream())                                # no norm: the average alone
        np.testing.assert_allclose(host(xo), x_ref, rtol=2e-5, atol=2e-5 * np.abs(x_ref).max())


@pytest.mark.parametrize("width", [1, 7, 36, 2052])
def test_shift_blends_in_rows_and_beside_the_norm(width):
    """The five blends from rows (F32 and split outputs) and one token at a time inside the norm launch: the same numbers, the carried row
    never read at position 0."""
    rng = np.random.default_rng(width)
    T, eps = 21, 1e-5
    X, g = rng.standard_normal((T, width)), 1 + 0.3 * rng.standard_normal(width)
    mu = rng.uniform(0, 1, (5, width))
    H = O.norm_groups(X, g, 1, eps)
    ref = [H + (O.shifted(H) - H) * m for m in mu]
    mus = [dev(m) for m in mu]
    for sizes in ([T], [1] * T, [2, 1, 7, 11]):
        carried, pos = dev(rng.standard_normal(width)), 0
        for n in sizes:
            out, sp = [torch.empty(n, width, device="cuda") for _ in range(5)], [split_buffer(n, width) for _ in range(5)]
            lib().nt_b200_shift_mix_rows(5, ptrs(mus), ptrs(out), ptrs(sp), dp(H[pos:pos + n]), carried.data_ptr(), n, width, pos, stream())
            for s in range(5):
                np.testing.assert_allclose(host(out[s]), ref[s][pos:pos + n], rtol=1e-5, atol=1e-6)
                np.testing.assert_allclose(joined(sp[s], n, width), ref[s][pos:pos + n], rtol=1e-4, atol=1e-4)
            pos += n
        np.testing.assert_allclose(host(carried), H[-1], rtol=1e-5, atol=1e-6)
    carried = dev(rng.standard_normal(width))
    for t in range(6):
        out, ho = [torch.empty(width, device="cuda") for _ in range(5)], torch.empty(width, device="cuda")
        lib().nt_b200_depth_norm_rows(dp(X[t]), width, 1, None, None, ho.data_ptr(), None, dp(g), eps, 1, width, 1, 5, ptrs(mus), ptrs(out), carried.data_ptr(), t, stream())
        np.testing.assert_allclose(host(ho), H[t], rtol=2e-5, atol=2e-5)
        for s in range(5):
            np.testing.assert_allclose(host(out[s]), ref[s][t], rtol=3e-5, atol=3e-5)


def wkv_inputs(rng, T, H, D, rank=None):
    r, k, v = (rng.standard_normal((T, H, D)) for _ in range(3))
    raw, w0, u = rng.standard_normal((T, H, D)), rng.uniform(-5, 1, (H, D)), rng.standard_normal((H, D))
    return r, k, v, raw, w0, u


def run_wkv_rows(r, k, v, raw, w0, u, sizes, rng, segments=False):
    T, H, D = r.shape
    scratch = torch.full((lib().nt_b200_wkv_scratch_floats(H, D),), float("nan"), device="cuda") if segments else None
    state = dev(rng.standard_normal((H, D, D)))                               # stale: a step at position 0 starts from zeros
    got, pos = [], 0
    for n in sizes:
        sl = slice(pos, pos + n)
        dr, dk, a, ruk, out = dev(r[sl]), dev(k[sl]), dev(raw[sl]), torch.empty(n, H, device="cuda"), torch.empty(n, H, D, device="cuda")
        lib().nt_b200_wkv_prep(a.data_ptr(), ruk.data_ptr(), dr.data_ptr(), dk.data_ptr(), dp(w0), dp(u), n, H, D, stream())
        lib().nt_b200_wkv_rows(out.data_ptr(), dr.data_ptr(), dk.data_ptr(), dp(v[sl]), a.data_ptr(), ruk.data_ptr(), state.data_ptr(), n, H, D, pos,
                               scratch.data_ptr() if segments else None, stream())
        got.append(host(out)); pos += n
    return np.concatenate(got)


@pytest.mark.parametrize("H,D", [(2, 1), (3, 7), (2, 8), (1, 16), (3, 17), (2, 32), (4, 33), (2, 64), (1, 100), (1, 127), (2, 128), (1, 200), (1, 255), (1, 256)])
def test_wkv_recurrence_and_state_hand_over(H, D):
    rng = np.random.default_rng(H * 1000 + D)
    T = 37
    r, k, v, raw, w0, u = wkv_inputs(rng, T, H, D)
    ref = O.wkv_recurrence(r, k, v, np.exp(-np.exp(raw + w0)), u)
    for sizes in ([T], [1] * T, [2, 16, 1, 15, 3]):
        np.testing.assert_allclose(run_wkv_rows(r, k, v, raw, w0, u, sizes, rng), ref, rtol=2e-4, atol=2e-5 * np.abs(ref).max())


@pytest.mark.parametrize("H,D", [(2, 5), (1, 16), (3, 64), (2, 33), (1, 128), (1, 256), (2, 20)])
def test_wkv_segments_side_by_side(H, D):
    """Long steps run as segments whose states are joined; steps that start later, that end inside a tile or a segment, and short ones between."""
    rng = np.random.default_rng(D)
    T = 1100
    r, k, v, raw, w0, u = wkv_inputs(rng, T, H, D)
    w0 -= 3.0                                                                 # slow decays: states cross many segments
    ref = O.wkv_recurrence(r, k, v, np.exp(-np.exp(raw + w0)), u)
    for sizes in ([T], [5, 1000, 95], [517, 583], [1024, 1, 75]):
        np.testing.assert_allclose(run_wkv_rows(r, k, v, raw, w0, u, sizes, rng, segments=True), ref, rtol=5e-4, atol=1e-4 * np.abs(ref).max())


def test_wkv_keeps_a_far_write_under_slow_decay_and_loses_it_under_fast():
    rng = np.random.default_rng(5)
    T, H, D = 700, 2, 8
    r, k, v, raw, _, u = wkv_inputs(rng, T, H, D)
    raw *= 0.1
    v[3] = 60.0
    for level, alive in ((-9.0, True), (1.0, False)):
        w0 = np.full((H, D), level)
        w = np.exp(-np.exp(raw + w0))
        ref = O.wkv_recurrence(r, k, v, w, u)
        v2 = v.copy(); v2[3] = 0.0
        moved = np.abs(ref[-1] - O.wkv_recurrence(r, k, v2, w, u)[-1]).max()
        assert (moved > 1.0) == alive
        for sizes in ([T], [4, 696], [600] + [1] * 100):
            np.testing.assert_allclose(run_wkv_rows(r, k, v, raw, w0, u, sizes, rng), ref, rtol=5e-4, atol=1e-4 * np.abs(ref).max())


@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
@pytest.mark.parametrize("H,D,rank", [(2, 1, 1), (3, 9, 5), (2, 20, 16), (2, 64, 64), (1, 128, 24), (2, 36, 7), (1, 256, 8), (1, 250, 40)])
def test_wkv_token_equals_the_rows(dt, H, D, rank):
    """The one-launch token form: second low-rank matrix, decay, recurrence, head norm and gate."""
    rng = np.random.default_rng(D * 10 + rank)
    T, eps, n = 9, 1e-5, H * D
    r, k, v, _, w0, u = wkv_inputs(rng, T, H, D)
    a1, W2 = np.tanh(rng.standard_normal((T, rank))), O.bf16_grid(rng.standard_normal((n, rank)) * rank ** -0.5)
    gate, norm = rng.standard_normal((T, n)), 1 + 0.3 * rng.standard_normal(n)
    w = np.exp(-np.exp(a1 @ W2.T + w0.reshape(-1))).reshape(T, H, D)
    o = O.wkv_recurrence(r, k, v, w, u)
    ref = O.rms(o, eps).reshape(T, n) * norm * O.silu(gate)
    state, w2 = dev(rng.standard_normal((H, D, D))), dev(W2, TORCH_DT[dt])
    for t in range(T):
        out = torch.empty(n, device="cuda")
        lib().nt_b200_wkv_token(out.data_ptr(), dp(r[t]), dp(k[t]), dp(v[t]), dp(gate[t]), dp(a1[t]), w2.data_ptr(), int(dt), dp(w0), dp(u), dp(norm), state.data_ptr(), eps,
                                rank, H, D, t, stream())
        np.testing.assert_allclose(host(out), ref[t], rtol=3e-4, atol=3e-4)
    out, sp = torch.empty(T, n, device="cuda"), split_buffer(T, n)
    lib().nt_b200_wkv_out_norm(out.data_ptr(), sp.data_ptr(), dp(o), dp(gate), dp(norm), eps, T, H, D, stream())
    np.testing.assert_allclose(host(out), ref, rtol=2e-5, atol=2e-5)
    np.testing.assert_allclose(joined(sp, T, n), ref, rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("T,cols", [(3, 1), (5, 7), (9, 64)])
def test_xielu_both_branches(T, cols):
    rng = np.random.default_rng(cols)
    z = rng.standard_normal((T, cols)) * np.exp(rng.uniform(-8, 3, (T, cols)))
    z[0, 0] = 0.0
    z[-1, -1] = -120.0
    for p, q in ((0.3, -0.7), (-2.0, 3.0), (25.0, 0.0)):
        ref = O.xielu(z, p, q)
        x, sp = dev(z), split_buffer(T, cols)
        lib().nt_b200_xielu_rows(x.data_ptr(), sp.data_ptr(), x.data_ptr(), dp(np.array([p, q])), T, cols, stream())      # in place
        np.testing.assert_allclose(host(x), ref, rtol=2e-5, atol=1e-7)
        np.testing.assert_allclose(joined(sp, T, cols), ref, rtol=1e-4, atol=1e-6)


@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
def test_products_with_an_input_per_matrix(dt):
    rng = np.random.default_rng(4)
    shapes = [(5, 64), (300, 64), (17, 33), (1, 1), (64, 2056), (9, 520)]
    acts, act = [0, 1, 0, 2, 2, 1], np.array([0.4, -0.3])
    Ws = [O.bf16_grid(rng.standard_normal(s) * s[1] ** -0.5) for s in shapes]
    xs = [rng.standard_normal(s[1]) for s in shapes]
    ref = [W @ x for W, x in zip(Ws, xs)]
    ref = [np.tanh(y) if a == 1 else O.xielu(y, *act) if a == 2 else y for y, a in zip(ref, acts)]
    dts = [dt, dt, dt, dt, dt, DType.F32]                                     # an F32 table beside 16-bit matrices
    Wd = [dev(W, TORCH_DT[d]) for W, d in zip(Ws, dts)]
    xd, yd, ap = [dev(x) for x in xs], [torch.empty(s[0], device="cuda") for s in shapes], dev(act)
    lib().nt_b200_gemv_multi(6, ptrs(Wd), ints([int(d) for d in dts]), ptrs(xd), ptrs(yd), ints([s[0] for s in shapes]), ints([s[1] for s in shapes]), ints(acts),
                             ptrs([ap] * 6), stream())
    for y, want in zip(yd, ref):
        np.testing.assert_allclose(host(y), want, rtol=2e-5, atol=2e-5)


@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
@pytest.mark.parametrize("out,K1,Ke,K2,E,top", [(36, 21, 12, 17, 5, 2), (1, 1, 1, 1, 1, 1), (64, 64, 1032, 0, 3, 3), (3000, 40, 16, 2048, 4, 1), (20000, 24, 8, 8, 2, 1), (10, 2056, 0, 64, 0, 0)])
def test_sum_of_products_with_routed_matrices(dt, out, K1, Ke, K2, E, top):
    rng = np.random.default_rng(out + K1)
    grid = lambda r, c: O.bf16_grid(rng.standard_normal((r, c)) * c ** -0.5)
    W1, x1, y0 = grid(out, K1), rng.standard_normal(K1), rng.standard_normal(out)
    ref = W1 @ x1
    w1 = dev(W1, TORCH_DT[dt])
    table, sel, wt, xe, tabs = None, None, None, None, []
    if top:
        Ws = [grid(out, Ke) for _ in range(E)]
        sel, wt, xe = rng.permutation(E)[:top], rng.uniform(0.1, 1, top), rng.standard_normal((top, Ke))
        ref = ref + sum(w * (Ws[s] @ x) for s, w, x in zip(sel, wt, xe))
        tabs = [dev(W, TORCH_DT[dt]) for W in Ws]
        table = torch.tensor([t.data_ptr() for t in tabs], device="cuda", dtype=torch.int64)
        seld = torch.from_numpy(sel.astype(np.int32)).cuda()
    W2 = None
    if K2:
        W2, x2 = grid(out, K2), rng.standard_normal(K2)
        ref = ref + W2 @ x2
        W2 = dev(W2, TORCH_DT[dt])
    for add in (0, 1):
        y = dev(y0)
        lib().nt_b200_gemv_sum(y.data_ptr(), out, int(dt), add, w1.data_ptr(), dp(x1), K1, table.data_ptr() if top else None, seld.data_ptr() if top else None,
                               dp(wt) if top else None, top, dp(xe) if top else None, Ke, W2.data_ptr() if K2 else None, dp(x2) if K2 else None, K2, stream())
        np.testing.assert_allclose(host(y), ref + add * y0, rtol=3e-5, atol=3e-5)


@pytest.mark.parametrize("E,top,scale", [(5, 2, 1.7), (1, 1, 1.0), (33, 33, 0.5), (256, 8, 2.5), (64, 3, 1.0)])
def test_router_weights_are_shares_of_all_experts(E, top, scale):
    rng = np.random.default_rng(E)
    T, W = 11, 52
    h, R = rng.standard_normal((T, W)), rng.standard_normal((E, W)) * 0.4
    sel_ref, wt_ref = O.route(h, R, top, scale)
    sel, wt = torch.zeros(T, top, device="cuda", dtype=torch.int32), torch.zeros(T, top, device="cuda")
    lib().nt_b200_moe_route_all(sel.data_ptr(), wt.data_ptr(), dp(h), dp(R), E, top, scale, W, T, stream())
    np.testing.assert_array_equal(sel.cpu().numpy(), sel_ref)
    np.testing.assert_allclose(host(wt), wt_ref, rtol=2e-5, atol=1e-7)
    if top < E:
        assert np.all(wt_ref.sum(1) < scale * 0.999999)                       # not renormalized
    # equal logits: the lowest indices are chosen, every share is 1 / E
    lib().nt_b200_moe_route_all(sel.data_ptr(), wt.data_ptr(), dp(np.zeros((T, W))), dp(R), E, top, scale, W, T, stream())
    np.testing.assert_array_equal(sel.cpu().numpy(), np.tile(np.arange(top), (T, 1)))
    np.testing.assert_allclose(host(wt), scale / E, rtol=1e-5)


@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
@pytest.mark.parametrize("E,top,ff,shared,W", [(5, 2, 12, 17, 36), (4, 4, 1, 0, 8), (40, 3, 64, 40, 128), (1, 1, 7, 1, 5)])
def test_choice_and_gated_experts_with_a_gated_shared_one(dt, E, top, ff, shared, W):
    rng = np.random.default_rng(E + ff)
    grid = lambda r, c: O.bf16_grid(rng.standard_normal((r, c)) * c ** -0.5)
    h, z, scale = rng.standard_normal(W), rng.standard_normal(E) * 2, 1.3
    Gs, Us, sg, su = [grid(ff, W) for _ in range(E)], [grid(ff, W) for _ in range(E)], grid(max(shared, 1), W), grid(max(shared, 1), W)
    s = np.exp(z - z.max()); s /= s.sum()
    order = np.argsort(-s, kind="stable")[:top]
    act_ref = np.concatenate([O.silu(Gs[e] @ h) * (Us[e] @ h) for e in order] + ([O.silu(sg @ h) * (su @ h)] if shared else []))
    g, u = [dev(a, TORCH_DT[dt]) for a in Gs], [dev(a, TORCH_DT[dt]) for a in Us]
    tab = lambda ts: torch.tensor([t.data_ptr() for t in ts], device="cuda", dtype=torch.int64)
    gt, ut = tab(g), tab(u)
    act, sel, wt = torch.zeros(top * ff + shared, device="cuda"), torch.zeros(top, device="cuda", dtype=torch.int32), torch.zeros(top, device="cuda")
    lib().nt_b200_moe_choose_up(act.data_ptr(), sel.data_ptr(), wt.data_ptr(), dp(h), dp(z), gt.data_ptr(), ut.data_ptr(), dp(sg, TORCH_DT[dt]), dp(su, TORCH_DT[dt]), int(dt),
                                E, top, scale, ff, shared, W, stream())
    np.testing.assert_array_equal(sel.cpu().numpy(), order)
    np.testing.assert_allclose(host(wt), s[order] * scale, rtol=1e-5)
    np.testing.assert_allclose(host(act), act_ref, rtol=3e-5, atol=3e-5)


# ---------------------------------------------------------------- windowed attention over shared rows
def rows_ref(Q, rows, vdim, scale, window, p0):
    """Q [T, H, D] at positions p0..; rows [S, >= D]: keys the first D numbers, values the first vdim."""
    T, H, D = Q.shape
    S = rows.shape[0]
    mask = O.window_mask(S, window or None)[p0:p0 + T]
    s = np.einsum("thd,sd->hts", Q, rows[:, :D]) * scale
    return np.einsum("hts,sv->thv", O.softmax_rows(s, mask[None]), rows[:, :vdim])


def run_rows(Q, rows, vdim, scale, window, dt, sizes, form):
    S, H, D = Q.shape
    cache, out, pos = dev(rows, TORCH_DT[dt]), [], 0
    for n in sizes:
        o = torch.empty(n, H, vdim, device="cuda")
        rc = lib().nt_b200_attention_rows_window(o.data_ptr(), dp(Q[pos:pos + n]), cache.data_ptr(), int(dt), n, pos, S, H, D, vdim, rows.shape[1], scale, window, form, stream())
        assert rc == 0
        out.append(host(o)); pos += n
    return np.concatenate(out)


@pytest.mark.parametrize("form", [0, 1])
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 31, 33, 64, 100, 500, 0])
def test_windowed_rows_attention(window, form):
    rng = np.random.default_rng(window)
    S, H, D, V = 130, 3, 40, 24
    Q, rows = rng.standard_normal((S, H, D)), O.bf16_grid(rng.standard_normal((S, D)))
    ref = rows_ref(Q, rows, V, D ** -0.5, window, 0)
    for dt in (DType.F32, DType.BF16):
        for sizes in ([S], [100] + [1] * 30, [2, 3, 17, 108]):
            np.testing.assert_allclose(run_rows(Q, rows, V, D ** -0.5, window, dt, sizes, form), ref, rtol=5e-5, atol=5e-5)


def loud(rng, S, H, D, at):
    """One key matches every query, all others do not: its value comes through wherever it is visible."""
    Q, K = rng.standard_normal((S, H, D)) * 0.1, rng.standard_normal((S, D)) * 0.1
    Q[:, :, 0] = 6.0
    K[:, 0] = 0.0
    K[at, 0] = 6.0
    return Q, K


@pytest.mark.parametrize("window", [16, 48, 129, 300])
@pytest.mark.parametrize("at", [0, 15, 16, 255, 311])
def test_a_loud_key_is_seen_inside_the_window_only(window, at):
    """Just inside and just outside the window's edge, at the borders of key groups, slices and tiles; prompt, portions and decoded tokens."""
    rng = np.random.default_rng(at)
    S, H, D, V = 700, 2, 64, 64
    Q, K = loud(rng, S, H, D, at)
    K[:, 1] = 0.0
    K[at, 1] = 40.0
    Q[:, :, 1] = 0.0
    ref = rows_ref(Q, K, V, 1.0, window, 0)
    inside, outside = at + window - 1, at + window
    assert ref[inside, :, 1].min() > 20.0 and np.abs(ref[outside, :, 1]).max() < 1.0 and (at == 0 or np.abs(ref[at - 1, :, 1]).max() < 1.0)
    for form in (0, 1):
        for sizes in ([S], [outside] + [1] * 2 + [S - outside - 2], [inside] + [1] * 3 + [S - inside - 3]):
            np.testing.assert_allclose(run_rows(Q, K, V, 1.0, window, DType.F32, sizes, form), ref, rtol=1e-4, atol=1e-3)
    # the tiled form over per-head keys and values, from every portion start; its first visible row is row 0 of what it is given
    kf = np.repeat(K[:, None, :], H, 1)
    kd, vd = dev(kf, torch.bfloat16), dev(kf, torch.bfloat16)
    b = O.bf16_grid(K)
    ref16 = rows_ref(Q, b, V, 1.0, window, 0)
    for p0, n in ((0, S), (inside - 3, 40), (outside, 17), (S - 64, 64)):
        lo = max(0, p0 - window + 1)
        o = torch.empty(n, H, V, device="cuda")
        lib().nt_b200_attention_heads_window(o.data_ptr(), dp(Q[p0:p0 + n]), kd.data_ptr() + lo * H * D * 2, vd.data_ptr() + lo * H * V * 2, n, p0 - lo, p0 + n - lo, H, D, V,
                                             1.0, window, stream())
        np.testing.assert_allclose(host(o), ref16[p0:p0 + n], rtol=2e-3, atol=2e-3)


# ---------------------------------------------------------------- whole models through the engine
def build(cfg, W, exact, max_context=256):
    return Model.from_config_json(cfg, device_tensors(W, exact), max_context=max_context, exact_f32=exact)


def run_portions(model, toks, sizes):
    rows, pos = [], 0
    for n in sizes:
        rows.append(model.forward_logits(toks[pos:pos + n], pos, list(range(n))))
        pos += n
    assert pos == len(toks)
    return np.concatenate(rows)


LA, WK = "latent_attention", "wkv"
CONFIGS = {
    "base": dict(),
    "attention_first_other_feed_forwards": dict(pattern=(LA, LA, WK), mlp=("dense", None, "moe"), groups=1, window=1),
    "recurrence_only": dict(pattern=(WK, WK, WK), mlp=("moe", None, "dense"), groups=9, shared=0, w_heads=4, w_dim=16),
    "no_window_top_of_all": dict(pattern=(LA, WK), mlp=("moe",), window=0, experts=4, top=4, router_scale=1.0, rot_dim=2, dim=5),
    "one_layer": dict(pattern=(LA,), mlp=("moe",), experts=3, top=1, window=2, shared=12, eff=12),
    "every_size_one": dict(pattern=(WK, LA), mlp=("dense", "moe"), width=1, vocab=5, groups=1, buckets=1, mul_prev=1, mul_cur=1, heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1,
                           w_heads=1, w_dim=1, rank=1, ff=1, experts=1, top=1, eff=1, shared=1, window=1),
    "unrotated_wide_latent": dict(pattern=(LA, WK), mlp=("dense", "moe"), rot_dim=0, dim=12, kv_rank=300, vdim=20, heads=5, window=30),
    "heads_wider_than_the_tiled_kernel": dict(pattern=(LA, WK), mlp=(None, "dense"), dim=180, rot_dim=20, vdim=130, heads=2, window=25, w_dim=40),
    # tile-aligned matrices: with BF16 weights the projections run on the tensor cores, short ones through padded copies, the attention on the tiled kernel
    "tensor_core_tiles": dict(width=128, vocab=128, groups=4, heads=2, dim=40, rot_dim=24, vdim=48, kv_rank=64, window=20, w_heads=4, w_dim=32, rank=64, ff=192, experts=4, top=2,
                              eff=128, shared=128),
    "tensor_core_tiles_ragged": dict(width=192, vocab=100, groups=6, heads=3, dim=64, rot_dim=32, vdim=80, kv_rank=96, window=37, w_heads=3, w_dim=64, rank=16, ff=320, experts=6,
                                     top=3, eff=64, shared=192),
}


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("exact", [True, False])
def test_model_schedules_agree_with_oracle(name, exact):
    rng = np.random.default_rng(len(name))
    cfg, W = O.random_model(rng, **CONFIGS[name])
    S = 61
    toks = rng.integers(0, cfg["vocab"], S).astype(np.int32)
    ref = O.forward(cfg, W, toks)
    m = build(cfg, W, exact)
    tol = 3e-4 if exact else 3e-2                                        # 16-bit cache rows in the second mode; everything else is F32 there too
    if cfg["width"] == 1:
        tol = 2e-2 if exact else 2e-1                                    # the norm of one channel is a sign: next to 0 it magnifies rounding
    whole = run_portions(m, toks, [S])
    assert rel_rms(whole, ref) < tol
    single = run_portions(m, toks, [1] * S)
    assert rel_rms(single, ref) < tol
    mixed = run_portions(m, toks, [2, 17, 3, 2, 20, 5, 1, 1, 8, 2])      # portions cut anywhere, in the middle of a window
    assert rel_rms(mixed, ref) < tol
    assert rel_rms(run_portions(m, toks, [40] + [1] * 21), ref) < tol
    if exact and cfg["width"] > 1:                                       # how a prompt is cut changes rounding only
        assert rel_rms(single, whole) < 1e-4 and rel_rms(mixed, whole) < 1e-4
    m.close()


def test_each_mechanism_in_a_model_of_its_own():
    """Models of one layer each, so that a fault names its mechanism."""
    for k, kw in enumerate((dict(pattern=(LA,), mlp=(None,)), dict(pattern=(WK,), mlp=(None,)), dict(pattern=(LA,), mlp=("dense",)), dict(pattern=(WK,), mlp=("moe",)),
                            dict(pattern=(WK,), mlp=("moe",), shared=0), dict(pattern=(LA, LA), mlp=(None,), groups=12))):
        rng = np.random.default_rng(k)
        cfg, W = O.random_model(rng, **kw)
        toks = rng.integers(0, cfg["vocab"], 30).astype(np.int32)
        m = build(cfg, W, True)
        ref = O.forward(cfg, W, toks)
        assert rel_rms(run_portions(m, toks, [30]), ref) < 1e-4, kw
        assert rel_rms(run_portions(m, toks, [1] * 30), ref) < 1e-4, kw
        m.close()


def test_first_tokens_and_single_token_request():
    rng = np.random.default_rng(2)
    cfg, W = O.random_model(rng)
    toks = rng.integers(0, cfg["vocab"], 5).astype(np.int32)
    ref = O.forward(cfg, W, toks)
    m = build(cfg, W, True)
    assert rel_rms(run_portions(m, toks[:1], [1]), ref[:1]) < 2e-4
    assert rel_rms(run_portions(m, toks, [2, 3]), ref) < 2e-4
    assert rel_rms(run_portions(m, toks, [1, 1, 1, 2]), ref) < 2e-4
    m.set_prefill_min_tokens(2)                                           # the same portions as prompt rows instead of decode steps
    assert rel_rms(run_portions(m, toks, [2, 3]), ref) < 2e-4
    assert rel_rms(run_portions(m, toks, [2, 1, 2]), ref) < 2e-4
    m.close()


@pytest.mark.parametrize("window", [3, 16, 17])
def test_short_prompt_portions_cross_window_edges(window):
    """Every portion runs as prompt rows (two at least), so the first row of each reads cache rows, the carried row and the previous token."""
    rng = np.random.default_rng(window)
    cfg, W = O.random_model(rng, window=window)
    S = 70
    toks = rng.integers(0, cfg["vocab"], S).astype(np.int32)
    ref = O.forward(cfg, W, toks)
    for exact in (True, False):
        m = build(cfg, W, exact)
        m.set_prefill_min_tokens(2)
        for sizes in ([2] * 35, [window + 1, window - 1, 2, S - 2 * window - 2], [3, 17, 16, 34]):
            assert rel_rms(run_portions(m, toks, sizes), ref) < (3e-4 if exact else 3e-2)
        m.close()


def test_rows_and_states_are_reused_between_requests():
    """A second request starts at position 0 over the first one's cache rows, matrix states, carried rows and previous token: bit-equal to
    running alone."""
    rng = np.random.default_rng(21)
    cfg, W = O.random_model(rng)
    a = rng.integers(0, cfg["vocab"], 50).astype(np.int32)
    b = rng.integers(0, cfg["vocab"], 30).astype(np.int32)
    for first in ([50], [20] + [1] * 30):
        m = build(cfg, W, True)
        run_portions(m, a, first)
        after_a = run_portions(m, b, [18] + [1] * 12)
        m2 = build(cfg, W, True)
        alone = run_portions(m2, b, [18] + [1] * 12)
        np.testing.assert_array_equal(after_a, alone)
        assert rel_rms(alone, O.forward(cfg, W, b)) < 2e-4
        after_a = run_portions(m, b[:3], [1, 1, 1])                      # and again, decoding from the very first token
        np.testing.assert_array_equal(after_a, run_portions(m2, b[:3], [1, 1, 1]))
        m.close(); m2.close()


def test_the_previous_token_crosses_every_kind_of_cut():
    """One WKV layer without feed-forward and blends of zero: only the pair embedding and the state connect positions.  Two prompts that
    differ in the token before the cut must differ behind it by the oracle's amount, whatever step kinds meet at the cut."""
    rng = np.random.default_rng(9)
    cfg, W = O.random_model(rng, pattern=(WK,), mlp=(None,), buckets=997, mul_prev=31, mul_cur=17)
    W["l0.mix.o"][:] = 0.0                                                # the pair embedding is the only path
    toks = rng.integers(0, cfg["vocab"], 60).astype(np.int32)
    other = toks.copy(); other[29] = (other[29] + 1) % cfg["vocab"]
    m = build(cfg, W, True)
    for t in (toks, other):
        ref = O.forward(cfg, W, t)
        for sizes in ([30, 30], [30] + [1] * 30, [1] * 30 + [30], [1] * 60, [28, 2, 30]):
            assert rel_rms(run_portions(m, t, sizes), ref) < 1e-4
    assert rel_rms(O.forward(cfg, W, other)[30:31], O.forward(cfg, W, toks)[30:31]) > 0.1
    m.close()


def test_prompt_longer_than_one_portion_of_the_engine():
    """2100 tokens: the engine cuts the prompt at 2048, so every state crosses that cut; 2049: the second part is a single row; tile-aligned
    sizes, both modes."""
    rng = np.random.default_rng(3)
    cfg, W = O.random_model(rng, **CONFIGS["tensor_core_tiles"])
    S = 2100
    toks = rng.integers(0, cfg["vocab"], S).astype(np.int32)
    ref = O.forward(cfg, W, toks)
    want = [0, 1, 63, 64, 2047, 2048, 2049, S - 1]
    for exact in (True, False):
        m = build(cfg, W, exact, max_context=2304)
        tol = 5e-4 if exact else 3e-2
        assert rel_rms(m.forward_logits(toks, 0, want), ref[want]) < tol
        assert rel_rms(m.forward_logits(toks[:2049], 0, want[:6]), ref[want[:6]]) < tol
        assert rel_rms(m.forward_logits(toks[2049:], 2049, [0, S - 2050]), ref[[2049, S - 1]]) < tol
        m.close()


def test_long_decode_and_graph_replay():
    rng = np.random.default_rng(8)
    cfg, W = O.random_model(rng, pattern=(WK, LA), mlp=("dense", "moe"), width=32, groups=4, vocab=50, window=40)
    S = 300
    toks = rng.integers(0, cfg["vocab"], S).astype(np.int32)
    ref = O.forward(cfg, W, toks)
    m = build(cfg, W, True, max_context=512)
    assert rel_rms(run_portions(m, toks, [3] + [1] * (S - 3)), ref) < 3e-4
    m.use_graph(False)
    m.clear_kv()
    assert rel_rms(run_portions(m, toks, [3] + [1] * (S - 3)), ref) < 3e-4
    m.close()


@pytest.mark.parametrize("kind", [LA, WK])
def test_a_far_token_reaches_as_far_as_its_mechanism_lets_it(kind):
    """One layer, so the mixer is the only path between positions.  Token 0 occurs once and shouts: through the window it must be heard
    up to the edge and not behind it; through the recurrence with a slow decay it must still be heard hundreds of tokens on."""
    rng = np.random.default_rng(13)
    window, S = 200, 420
    cfg, W = O.random_model(rng, pattern=(kind,), mlp=(None,), window=window, groups=1, rot_dim=6, scale=2.0)
    W["embed"][0] *= 8.0
    W["bigram"][:] *= 0.01                                                 # the token itself, not the pair, is what the layer hears
    if kind == WK:
        W["l0.mix.w0"][:] = -9.0
        W["l0.mix.w2"][:] *= 0.1
        W["l0.mix.mu.k"][:] = 0.0; W["l0.mix.mu.v"][:] = 0.0
    toks = rng.integers(1, cfg["vocab"], S).astype(np.int32)
    base = O.forward(cfg, W, toks)
    m = build(cfg, W, True, max_context=512)
    for at in (0, 5, 16):
        t = toks.copy(); t[at] = 0
        ref = O.forward(cfg, W, t)
        moved = np.sqrt(((ref - base) ** 2).mean(1))
        if kind == LA:
            # the pair embedding of the next token hears it too: position at + window still sees that one, the next sees neither
            assert moved[at + 2:at + window + 1].min() > 0 and moved[at + window + 1:].max() < 1e-9
        else:
            assert moved[-1] > 1e-4
        for sizes in ([S], [at + window - 1] + [1] * 3 + [S - at - window - 2], [3, 300] + [1] * (S - 303)):
            assert rel_rms(run_portions(m, t, sizes), ref) < 3e-4
    m.close()


def test_greedy_generation_through_the_engine(tmp_path):
    rng = np.random.default_rng(4)
    cfg, W = O.random_model(rng)
    for L in cfg["layers"]:                                                   # the folder states no rank: the tensors' shapes give it
        if L["type"] == WK:
            del L["mixer"]["decay_rank"]
    d = write_model_dir(tmp_path / "m", cfg, W)
    prompt = rng.integers(0, cfg["vocab"], 19).astype(np.int32)
    for exact in (True, False):
        e = Engine()
        assert e.load_path(d, max_context=128, exact_f32=exact)
        assert e.vocab_size == cfg["vocab"] and e.n_layers == 4
        new = e.generate_ids(prompt, max_tokens=24, temperature=0.0)
        assert len(new) == 24
        assert e.generate_ids(prompt, max_tokens=24, temperature=0.0) == new       # rows and states are taken over from position 0
        logits = O.forward(cfg, W, np.concatenate([prompt, np.asarray(new, dtype=np.int32)]))
        for i, tok in enumerate(new):                                         # every generated id is the oracle's greedy choice
            row = logits[len(prompt) - 1 + i]
            assert row[tok] >= row.max() - (1e-3 if exact else 0.2), (exact, i)
        sampled = e.generate_ids(prompt, max_tokens=8, temperature=0.8, top_k=10, top_p=0.9, repeat_penalty=1.1, seed=7)
        assert len(sampled) == 8 and all(0 <= s < cfg["vocab"] for s in sampled)
        e.close()


def test_model_folder_loads_like_device_tensors(tmp_path):
    rng = np.random.default_rng(6)
    cfg, W = O.random_model(rng)
    toks = rng.integers(0, cfg["vocab"], 33).astype(np.int32)
    a = Model.load_dir(write_model_dir(tmp_path / "m", cfg, W), max_context=64, exact_f32=True)
    b = build(cfg, W, True, max_context=64)
    np.testing.assert_array_equal(a.forward_logits(toks, 0, [0, 5, 32]), b.forward_logits(toks, 0, [0, 5, 32]))
    a.close(); b.close()
