"""Tibelix on the GPU against the plain float64 oracle (tests/tibelix_oracle.py): each mechanism's kernel alone, then whole models through the
engine's step function — prompt pass vs token-by-token decoding, portions down to two tokens, cache rows and states reused by a second
request, keys far away and at tile and slice borders, steps of the query temperature, the first tokens, sizes that are odd, 1 or equal where the
usual ones differ, long decoding with and without graph replay, and greedy generation through the engine's entry point."""
import ctypes as C

import numpy as np
import pytest
import torch

import tibelix_oracle as O
from tibelix_util import device_tensors
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


def joined(split, rows, cols):
    """hi + lo of a BF16 split workspace, the live rows."""
    mp = (rows + 127) // 128 * 128
    w = split.view(torch.bfloat16).reshape(2, mp, cols)
    return host(w[0, :rows]) + host(w[1, :rows])


def split_buffer(rows, cols):
    return torch.zeros(2 * ((rows + 127) // 128 * 128) * cols, device="cuda", dtype=torch.bfloat16)


# ---------------------------------------------------------------- row kernels alone
@pytest.mark.parametrize("width", [1, 7, 36, 130, 1024, 2048, 2052, 4100, 5003, 8192, 16384, 20000])
@pytest.mark.parametrize("rows", [1, 5])
def test_norms_around_a_sublayer(width, rows):
    rng = np.random.default_rng(width + rows)
    eps = 1e-3
    x, y = rng.standard_normal((rows, width)), rng.standard_normal((rows, width)) * 3
    gy, gh = 1 + 0.3 * rng.standard_normal(width), 1 + 0.3 * rng.standard_normal(width)
    for with_y in (True, False):
        x_ref = x + O.norm_plain(y, gy, eps) if with_y else x
        h_ref = O.norm_plain(x_ref, gh, eps)
        xd, h, sp = dev(x), torch.empty(rows, width, device="cuda"), split_buffer(rows, width)
        lib().nt_b200_sandwich_norm_rows(xd.data_ptr(), dp(y) if with_y else None, dp(gy), dp(gh), h.data_ptr(), sp.data_ptr(), rows, width, eps, stream())
        np.testing.assert_allclose(host(xd), x_ref, rtol=2e-5, atol=2e-5)
        np.testing.assert_allclose(host(h), h_ref, rtol=3e-5, atol=3e-5)
        np.testing.assert_allclose(joined(sp, rows, width), h_ref, rtol=1e-4, atol=1e-4)
    xd = dev(x)
    lib().nt_b200_sandwich_norm_rows(xd.data_ptr(), dp(y), dp(gy), None, None, None, rows, width, eps, stream())      # the last layer: no next input
    np.testing.assert_allclose(host(xd), x + O.norm_plain(y, gy, eps), rtol=2e-5, atol=2e-5)


@pytest.mark.parametrize("T,heads,per,ld", [(3, 2, 5, 2), (5, 4, 8, 128), (1, 3, 1, 3), (9, 40, 1, 40), (17, 12, 1, 128), (4, 3, 96, 3), (2, 1, 7, 4)])
def test_output_gates_by_head_and_by_channel(T, heads, per, ld):
    rng = np.random.default_rng(T)
    o, g = rng.standard_normal((T, heads * per)), rng.standard_normal((T, ld)) * 3
    ref = o * np.repeat(O.sigmoid(g[:, :heads]), per, axis=1)
    d, sp = dev(o), split_buffer(T, heads * per)
    lib().nt_b200_sigmoid_gate_rows(d.data_ptr(), sp.data_ptr(), d.data_ptr(), dp(g), ld, per, T, heads * per, stream())      # in place
    np.testing.assert_allclose(host(d), ref, rtol=1e-5, atol=1e-6)
    np.testing.assert_allclose(joined(sp, T, heads * per), ref, rtol=1e-4, atol=1e-5)


@pytest.mark.parametrize("M,N,K", [(1, 128, 64), (130, 256, 128), (77, 200, 192), (300, 512, 256)])
def test_squared_relu_in_rows_and_in_the_product(M, N, K):
    rng = np.random.default_rng(N)
    A, W = rng.standard_normal((M, K)), O.bf16_grid(rng.standard_normal((N, K)) * K ** -0.5)
    ref = np.maximum(A @ W.T, 0) ** 2
    z, sp = dev(A @ W.T), split_buffer(M, N)
    lib().nt_b200_relu2_rows(z.data_ptr(), sp.data_ptr(), z.data_ptr(), M, N, stream())
    np.testing.assert_allclose(host(z), ref, rtol=1e-5, atol=1e-6)
    np.testing.assert_allclose(joined(sp, M, N), ref, rtol=1e-4, atol=1e-5)
    sp.zero_()
    ws = split_buffer(M, K)
    assert lib().nt_b200_gemm_relu2(sp.data_ptr(), dp(A), dp(W, torch.bfloat16), M, N, K, ws.data_ptr(), stream()) == 0
    np.testing.assert_allclose(joined(sp, M, N), ref, rtol=1e-3, atol=2e-4 * ref.max())


def ptrs(ts):
    return (C.c_void_p * len(ts))(*[t.data_ptr() for t in ts])


@pytest.mark.parametrize("M,K,Ns", [(1, 64, [256, 260]), (130, 128, [512, 320, 256]), (300, 192, [256] * 6), (77, 64, [1000])])
def test_several_products_of_the_same_rows_in_one_launch(M, K, Ns):
    rng = np.random.default_rng(M)
    A = rng.standard_normal((M, K))
    Ws = [O.bf16_grid(rng.standard_normal((n, K)) * K ** -0.5) for n in Ns]
    Wd, Cd, ws = [dev(W, torch.bfloat16) for W in Ws], [torch.full((M + 1, n), 7.0, device="cuda") for n in Ns], split_buffer(M, K)
    rc = lib().nt_b200_gemm_multi(ptrs(Cd), dp(A), ptrs(Wd), (C.c_int * len(Ns))(*Ns), len(Ns), M, K, ws.data_ptr(), stream())
    assert rc == 0
    for c, W in zip(Cd, Ws):
        np.testing.assert_allclose(host(c)[:M], A @ W.T, rtol=1e-3, atol=2e-4)
        assert (host(c)[M] == 7.0).all()                                      # nothing behind the live rows
    assert lib().nt_b200_gemm_multi(ptrs(Cd[:1]), dp(A), ptrs(Wd[:1]), (C.c_int * 1)(128), 1, M, K, ws.data_ptr(), stream()) == -1      # too narrow


@pytest.mark.parametrize("width,experts", [(4, 1), (36, 5), (1024, 3), (2048, 16), (4100, 100), (8192, 256), (16384, 7)])
def test_norms_around_a_sublayer_with_the_routers_logits(width, experts):
    rng = np.random.default_rng(width)
    eps = 1e-3
    x, y, gy, gh = rng.standard_normal((1, width)), rng.standard_normal((1, width)) * 3, 1 + 0.3 * rng.standard_normal(width), 1 + 0.3 * rng.standard_normal(width)
    R = rng.standard_normal((experts, width)) * width ** -0.5
    x_ref = x + O.norm_plain(y, gy, eps)
    h_ref = O.norm_plain(x_ref, gh, eps)
    xd, xo, h, z = dev(x), torch.empty(1, width, device="cuda"), torch.empty(1, width, device="cuda"), torch.empty(experts, device="cuda")
    assert lib().nt_b200_sandwich_norm_router(xo.data_ptr(), xd.data_ptr(), dp(y), dp(gy), dp(gh), h.data_ptr(), dp(R), z.data_ptr(), experts, width, eps, stream()) == 0
    np.testing.assert_allclose(host(xo), x_ref, rtol=2e-5, atol=2e-5)
    np.testing.assert_allclose(host(h), h_ref, rtol=3e-5, atol=3e-5)
    np.testing.assert_allclose(host(z), (R @ h_ref[0]), rtol=1e-4, atol=1e-4)
    np.testing.assert_array_equal(host(xd), host(dev(x)))
    assert lib().nt_b200_sandwich_norm_router(xo.data_ptr(), xd.data_ptr(), dp(y), dp(gy), dp(gh), h.data_ptr(), dp(R), z.data_ptr(), experts, 7, eps, stream()) == -1


@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
@pytest.mark.parametrize("out,K", [(5, 13), (300, 64), (1, 1), (64, 1544), (2000, 768)])
def test_a_product_of_a_normed_input(dt, out, K):
    rng = np.random.default_rng(K)
    W, x, g = O.bf16_grid(rng.standard_normal((out, K)) * K ** -0.5), rng.standard_normal((1, K)) * 5, 1 + 0.3 * rng.standard_normal(K)
    y = torch.empty(out, device="cuda")
    lib().nt_b200_gemv_normed(y.data_ptr(), dp(W, TORCH_DT[dt]), int(dt), dp(x), dp(g), 1e-2, out, K, stream())
    np.testing.assert_allclose(host(y), W @ O.norm_plain(x, g, 1e-2)[0], rtol=3e-5, atol=3e-5)


# ---------------------------------------------------------------- attention
@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
@pytest.mark.parametrize("H,G,D,V,every", [(2, 1, 8, 5, 4), (6, 3, 10, 7, 1), (1, 1, 1, 1, 7), (4, 2, 96, 64, 16), (3, 3, 33, 130, 1000), (2, 2, 7, 7, 2.5)])
def test_unit_heads_and_query_temperature(dt, H, G, D, V, every):
    """Positions around every step of the temperature; a layer that reads another layer's rows prepares its queries only."""
    rng = np.random.default_rng(H * 100 + D)
    p0, T, eps, coef = 5, 29, 1e-2, 0.8
    q, k, v = rng.standard_normal((T, H, D)) * 4, rng.standard_normal((T, G, D)) * 0.2, rng.standard_normal((T, G, V))
    temp = O.query_temperature(range(p0, p0 + T), coef, every)
    ref_q, ref_k = O.rms(q, eps) * temp[:, None, None], O.rms(k, eps)
    for with_k in (True, False):
        qd = dev(q)
        kc, vc = torch.zeros(p0 + T + 3, G, D, device="cuda", dtype=TORCH_DT[dt]), torch.zeros(p0 + T + 3, G, V, device="cuda", dtype=TORCH_DT[dt])
        lib().nt_b200_head_prep_unit(qd.data_ptr(), dp(k) if with_k else None, dp(v) if with_k else None, H, G, D, V, eps, coef, every, kc.data_ptr(), vc.data_ptr(), int(dt), T, p0,
                                     stream())
        np.testing.assert_allclose(host(qd), ref_q, rtol=2e-5, atol=1e-5)
        tol = dict(rtol=2e-5, atol=1e-6) if dt == DType.F32 else dict(rtol=8e-3, atol=1e-3)
        np.testing.assert_allclose(host(kc)[p0:p0 + T], ref_k * with_k, **tol)
        np.testing.assert_allclose(host(vc)[p0:p0 + T], v * with_k, **tol)
        assert host(kc)[:p0].any() == 0 and host(vc)[p0 + T:].any() == 0
    qd = dev(q)
    lib().nt_b200_head_prep_unit(qd.data_ptr(), None, None, H, G, D, V, eps, coef, 0.0, kc.data_ptr(), vc.data_ptr(), int(dt), T, p0, stream())      # no temperature
    np.testing.assert_allclose(host(qd), O.rms(q, eps), rtol=2e-5, atol=1e-5)


def run_biased(q, k, v, scale, slopes, gate, dt, sizes, max_seq=None, unit_sink=True):
    """q [S, H, D] over cache rows k, v [S, G, .], in portions."""
    S, H, D = q.shape
    G, V = v.shape[1:]
    n_rows = max_seq or S
    kc, vc = torch.zeros(n_rows, G, D, device="cuda", dtype=TORCH_DT[dt]), torch.zeros(n_rows, G, V, device="cuda", dtype=TORCH_DT[dt])
    kc[:S], vc[:S] = dev(k, TORCH_DT[dt]), dev(v, TORCH_DT[dt])
    out, pos = [], 0
    zeros = dp(np.zeros(H)) if unit_sink else None
    for n in sizes:
        o = torch.empty(n, H, V, device="cuda")
        lib().nt_b200_attention_biased(o.data_ptr(), dp(q[pos:pos + n]), kc.data_ptr(), vc.data_ptr(), int(dt), n, pos, n_rows, H, G, D, V, scale,
                                       dp(slopes) if slopes is not None else None, zeros, dp(gate[pos:pos + n]) if gate is not None else None, stream())
        out.append(host(o)); pos += n
    return np.concatenate(out)


@pytest.mark.parametrize("H,G,D,V", [(2, 1, 8, 5), (6, 3, 10, 7), (1, 1, 1, 1), (4, 2, 64, 64), (4, 1, 96, 96), (2, 2, 128, 128), (3, 1, 32, 64), (2, 1, 64, 128), (2, 2, 20, 300), (8, 8, 16, 16)])
def test_distance_bias_unit_sink_and_head_gate(H, G, D, V):
    rng = np.random.default_rng(H * 100 + D)
    S = 150
    q, k, v = rng.standard_normal((S, H, D)), O.bf16_grid(rng.standard_normal((S, G, D))), O.bf16_grid(rng.standard_normal((S, G, V)))
    gate = rng.standard_normal((S, H)) * 2
    for slopes in (O.slopes(H), np.zeros(H)):
        plain = O.biased_attention(q, k, v, D ** -0.5, slopes)
        gated = plain * O.sigmoid(gate)[:, :, None]
        for dt in (DType.F32, DType.BF16):
            for sizes in ([S], [120] + [1] * 30, [2, 3, 17, 128]):
                tol = 5e-5 if dt == DType.F32 else 5e-4                       # the tiled form's 16-bit operand pairs
                np.testing.assert_allclose(run_biased(q, k, v, D ** -0.5, slopes, None, dt, sizes), plain, rtol=tol, atol=tol)
                np.testing.assert_allclose(run_biased(q, k, v, D ** -0.5, slopes, gate, dt, sizes), gated, rtol=tol, atol=tol)
            # a decoded token over a long cache: its keys are split over a cluster
            np.testing.assert_allclose(run_biased(q, k, v, D ** -0.5, slopes, gate, dt, [149, 1], max_seq=3000), gated, rtol=5e-4, atol=5e-4)


@pytest.mark.parametrize("at", [0, 31, 32, 63, 64, 255, 256])
@pytest.mark.parametrize("D", [48, 64, 96])
def test_a_far_key_outweighs_the_bias_by_exactly_its_distance(at, D):
    """One key's score stands out by B.  Under a slope s it carries weight e^(B - s d) against the sink's 1 and nothing else: at every distance d,
    through tile, slice and cluster borders, in prompts and decoded."""
    rng = np.random.default_rng(at)
    S, H, B, slope = 700, 2, 30.0, np.array([0.04, 0.2])
    q, k, v = np.zeros((S, H, D)), np.zeros((S, 1, D)), np.zeros((S, 1, D))
    q[:, :, 0] = 1.0
    k[:, 0, 0] = -200.0                                                       # every other key is out of reach
    k[at, 0, 0] = B
    v[at, 0, 1] = 8.0
    ref = O.biased_attention(q, k, v, 1.0, slope)
    d = np.arange(S)[at:, None] - at
    np.testing.assert_allclose(ref[at:, :, 1], 8.0 / (1.0 + np.exp(slope * d - B)), rtol=1e-9)
    assert ref[-1, 0, 1] > 4.0 and (S - at < 300 or ref[-1, 1, 1] < 1e-6)      # one head still hears it at the end, the other no more
    for dt in (DType.F32, DType.BF16):
        for sizes in ([S], [at + 100] + [1] * 60 + [S - at - 160], [S - 40] + [1] * 40):
            np.testing.assert_allclose(run_biased(q, k, v, 1.0, slope, None, dt, sizes), ref, rtol=2e-3 if dt == DType.BF16 else 2e-4, atol=2e-4)
    assert not np.allclose(run_biased(q, k, v, 1.0, slope, None, DType.F32, [S], unit_sink=False), ref, atol=1e-2)      # the sink shows


@pytest.mark.parametrize("H,G,D,V", [(2, 1, 16, 16), (6, 2, 48, 32), (4, 4, 64, 64), (16, 4, 128, 128), (20, 1, 96, 96), (32, 1, 64, 512), (17, 1, 32, 144), (8, 1, 320, 256), (32, 1, 576, 512)])
@pytest.mark.parametrize("joint", [False, True])
def test_one_decoded_token_with_the_heads_of_a_key_head_together(H, G, D, V, joint):
    """Positions at the first token, around tile borders and where slices wrap over several tiles; distance bias, sink and gate on and off; a window;
    values in rows of their own or at the start of the key rows."""
    if (joint and (G > 1 or V > D)) or (not joint and D + V > 1000):
        pytest.skip("values at the start of the key rows: one key head, values no wider than the keys; the widest rows fit shared memory in that form only")
    rng = np.random.default_rng(H + D)
    S, max_seq, scale = 700, 1024, D ** -0.5
    k = O.bf16_grid(rng.standard_normal((S, G, D)))
    v = k[:, :, :V] if joint else O.bf16_grid(rng.standard_normal((S, G, V)))
    kc = dev(k, torch.bfloat16)
    vc = kc if joint else dev(v, torch.bfloat16)
    scratch = torch.full((lib().nt_b200_attention_rows_decode_scratch_floats(H, V),), float("nan"), device="cuda")
    slopes, zeros = O.slopes(H), np.zeros(H)
    for pos in (0, 1, 15, 62, 63, 64, 65, 127, 128, 500, 699):
        q, gate = rng.standard_normal((1, H, D)), rng.standard_normal(H)
        for window, seq, full in ((0, max_seq, True), (0, 64, False), (37, max_seq, False), (64, max_seq, True), (300, max_seq, False)):
            lo = max(0, pos + 1 - window) if window else 0
            ref = np.zeros((H, V))
            for h in range(H):
                g = h // (H // G)
                s = k[lo:pos + 1, g] @ q[0, h] * scale - full * slopes[h] * (pos - np.arange(lo, pos + 1))
                ones = np.ones((1, len(s)), dtype=bool)
                ref[h] = (O.sink_softmax(s[None], ones) if full else O.softmax_rows(s[None], ones))[0] @ v[lo:pos + 1, g] * (O.sigmoid(gate[h]) if full else 1.0)
            out = torch.empty(H, V, device="cuda")
            rc = lib().nt_b200_attention_rows_decode(out.data_ptr(), dp(q), kc.data_ptr(), vc.data_ptr(), pos, seq, H, G, D, V, G * D, G * D if joint else G * V, scale, window,
                                                     dp(slopes) if full else None, dp(zeros) if full else None, dp(gate) if full else None, scratch.data_ptr(), stream())
            assert rc == 0
            np.testing.assert_allclose(host(out), ref, rtol=3e-4, atol=3e-4)


def table64(rot):
    sc = rot.get("scaling")
    f = np.zeros(max(1, rot["dims"] // 2))
    mag = lib().nt_b200_rotary_table64(f.ctypes.data_as(C.c_void_p), rot["dims"], rot["base"], *((sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc else (0.0,) * 4))
    return torch.from_numpy(f).cuda(), mag


@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
@pytest.mark.parametrize("H,D,R,dims,rank,q_rank,p0", [(3, 9, 6, 6, 11, 13, 0), (1, 4, 2, 2, 1, 1, 1000), (2, 40, 24, 16, 64, 20, 37), (5, 8, 32, 32, 40, 96, 4000)])
def test_latent_rows_and_queries_under_the_long_context_blend(dt, H, D, R, dims, rank, q_rank, p0):
    rng = np.random.default_rng(D)
    T, eps, rot = 19, 1e-5, {"dims": dims, "base": 30000.0, "scaling": {"factor": 5.0, "original": 200, "fast": 16.0, "slow": 1.5}}
    freq, mag = table64(rot)
    cq, gq, dkv, gk = rng.standard_normal((T, q_rank)), 1 + 0.2 * rng.standard_normal(q_rank), rng.standard_normal((T, rank + R)) * 2, 1 + 0.2 * rng.standard_normal(rank)
    q, Wk = rng.standard_normal((T, H, D + R)), O.bf16_grid(rng.standard_normal((H * D, rank)) * D ** -0.5)
    pos = np.arange(p0, p0 + T)
    c, kr = O.norm_plain(dkv[:, :rank], gk, eps), O.rotate_pairs(dkv[:, rank:], pos, rot)
    qr = O.rotate_pairs(q[:, :, D:], pos, rot)
    cache, CQ = torch.zeros(p0 + T, rank + R, device="cuda", dtype=TORCH_DT[dt]), dev(cq)
    kw = (D + R + 15) // 16 * 16
    qa, qp = torch.empty(T, H, rank + R, device="cuda"), torch.empty(T, H, kw, device="cuda")
    lib().nt_b200_latent_rotated(CQ.data_ptr(), q_rank, dp(gq), dp(dkv), rank, R, dp(gk), eps, cache.data_ptr(), int(dt), dims, 1, freq.data_ptr(), mag, T, p0, qa.data_ptr(), dp(q),
                                 dp(Wk, TORCH_DT[dt]), int(dt), H, D, qp.data_ptr(), kw, stream())
    tol = dict(rtol=3e-5, atol=3e-5) if dt == DType.F32 else dict(rtol=8e-3, atol=8e-3)
    np.testing.assert_allclose(host(CQ), O.norm_plain(cq, gq, eps), rtol=2e-5, atol=2e-5)
    np.testing.assert_allclose(host(cache)[p0:], np.concatenate([c, kr], 1), **tol)
    want = np.concatenate([np.einsum("thd,hdr->thr", q[:, :, :D], Wk.reshape(H, D, rank)), qr], 2)
    np.testing.assert_allclose(host(qa), want, rtol=3e-5, atol=5e-5)
    np.testing.assert_allclose(host(qp)[:, :, :D + R], np.concatenate([q[:, :, :D], qr], 2), rtol=3e-5, atol=3e-5)
    assert not host(qp)[:, :, D + R:].any()


@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
def test_latent_values_with_an_output_gate(dt):
    rng = np.random.default_rng(3)
    for T, H, V, r in ((1, 3, 7, 11), (9, 2, 40, 64), (1, 1, 1, 1)):
        ol, Wv, g = rng.standard_normal((T, H, r)), O.bf16_grid(rng.standard_normal((H * V, r)) * r ** -0.5), rng.standard_normal((T, H * V)) * 3
        out = torch.empty(T, H * V, device="cuda")
        lib().nt_b200_latent_v_up_gated(out.data_ptr(), dp(ol), dp(Wv, TORCH_DT[dt]), int(dt), T, H, V, r, dp(g), stream())
        ref = np.einsum("thr,hvr->thv", ol, Wv.reshape(H, V, r)).reshape(T, H * V) * O.sigmoid(g)
        np.testing.assert_allclose(host(out), ref, rtol=3e-5, atol=3e-5)


@pytest.mark.parametrize("dt", [DType.F32, DType.BF16])
@pytest.mark.parametrize("H,D,R,V,r,p0", [(3, 9, 8, 7, 16, 0), (2, 40, 16, 48, 64, 37), (5, 8, 8, 33, 40, 300), (20, 16, 32, 64, 480, 130), (1, 4, 8, 1, 8, 5)])
def test_a_decoded_token_of_the_latent_attention(dt, H, D, R, V, r, p0):
    """Absorbed queries with the cache row on the way, slices, merge with the gated values."""
    rng = np.random.default_rng(r)
    eps, rot, S = 1e-5, {"dims": R, "base": 700.0}, p0 + 1
    c, kr = O.bf16_grid(rng.standard_normal((S, r))), O.bf16_grid(rng.standard_normal((S, R)))
    dkv, gk, q, g = rng.standard_normal((1, r + R)), 1 + 0.2 * rng.standard_normal(r), rng.standard_normal((1, H, D + R)), rng.standard_normal((1, H * V)) * 2
    Wk, Wv = O.bf16_grid(rng.standard_normal((H * D, r)) * r ** -0.5), O.bf16_grid(rng.standard_normal((H * V, r)) * r ** -0.5)
    cache = dev(np.concatenate([c, kr], 1), TORCH_DT[dt])
    cache[p0] = 99.0                                                          # overwritten by the token's own row
    out, scale = torch.empty(H * V, device="cuda"), (D + R) ** -0.5
    rc = lib().nt_b200_latent_token(out.data_ptr(), dp(q), dp(dkv), dp(gk), eps, cache.data_ptr(), int(dt), dp(Wk, TORCH_DT[dt]), dp(Wv, TORCH_DT[dt]), int(dt), p0, 1000, H, D, R, V, r, R,
                                    700.0, scale, dp(g), stream())
    assert rc == 0
    own = np.concatenate([O.norm_plain(dkv[:, :r], gk, eps), O.rotate_pairs(dkv[:, r:], [p0], rot)], 1)
    np.testing.assert_allclose(host(cache)[p0:], own, **(dict(rtol=3e-5, atol=3e-5) if dt == DType.F32 else dict(rtol=8e-3, atol=8e-3)))
    rows = host(cache)
    k, v = np.einsum("sr,hdr->shd", rows[:, :r], Wk.reshape(H, D, r)), np.einsum("sr,hvr->shv", rows[:, :r], Wv.reshape(H, V, r))
    qr = O.rotate_pairs(q[:, :, D:], [p0], rot)
    s = (np.einsum("hd,shd->hs", q[0, :, :D], k) + np.einsum("hd,sd->hs", qr[0], rows[:, r:])) * scale
    ref = np.einsum("hs,shv->hv", O.softmax_rows(s, np.ones_like(s, dtype=bool)), v).reshape(-1) * O.sigmoid(g[0])
    np.testing.assert_allclose(host(out), ref, rtol=2e-4, atol=1e-4)


# ---------------------------------------------------------------- matrix memory
def memory_inputs(rng, T, H, D, V, bias=(0.0, 2.0), spread=2.0):
    q, k, v = rng.standard_normal((T, H, D)), rng.standard_normal((T, H, D)) * D ** -0.5, rng.standard_normal((T, H, V))
    zi, zf = rng.standard_normal((T, H)) * spread, rng.standard_normal((T, H)) * spread
    return q, k, v, zi, zf, np.full(H, bias[0]) + 0.1 * rng.standard_normal(H), np.full(H, bias[1]) + 0.1 * rng.standard_normal(H)


def memory_ref(q, k, v, zi, zf, bi, bf, cap):
    i, f = O.mlstm_gates(zi + bi, zf + bf, cap)
    return O.mlstm_memory(q * q.shape[2] ** -0.5, k, v, i, f)


class Memory:
    """State of one sequence on the device, stale at first: a step at position 0 starts from zeros."""

    def __init__(self, rng, H, D, V, segments=False):
        self.state, self.m = dev(rng.standard_normal((H, V + 1, D))), dev(rng.standard_normal(H) * 5)
        self.scratch = torch.full((lib().nt_b200_mlstm_scratch_floats(H, D, V),), float("nan"), device="cuda") if segments else None

    def rows(self, q, k, v, zi, zf, bi, bf, cap, pos, ld=None):
        n, H, D = q.shape
        V = v.shape[2]
        a, b, em, den = (torch.empty(n, H, device="cuda") for _ in range(4))
        o = torch.empty(n, H, V, device="cuda")
        z = np.zeros((n, ld or 2 * H))
        z[:, :H], z[:, H:2 * H] = zi, zf
        zd = dev(z)
        _KEPT.append(zd)
        lib().nt_b200_mlstm_gates(a.data_ptr(), b.data_ptr(), em.data_ptr(), zd.data_ptr(), zd.data_ptr() + 4 * H, z.shape[1], dp(bi), dp(bf), cap, self.m.data_ptr(), n, H, pos, stream())
        lib().nt_b200_mlstm_rows(o.data_ptr(), den.data_ptr(), dp(q), dp(k), dp(v), a.data_ptr(), b.data_ptr(), self.state.data_ptr(), D ** -0.5, n, H, D, V, pos,
                                 self.scratch.data_ptr() if self.scratch is not None else None, stream())
        _KEPT.extend([a, b])
        return o, den, em


def run_memory(x, cap, sizes, rng, segments=False, ld=None):
    q, k, v, zi, zf, bi, bf = x
    mem = Memory(rng, q.shape[1], q.shape[2], v.shape[2], segments)
    got, pos = [], 0
    for n in sizes:
        sl = slice(pos, pos + n)
        o, den, em = mem.rows(q[sl], k[sl], v[sl], zi[sl], zf[sl], bi, bf, cap, pos, ld)
        got.append(host(o) / (np.maximum(np.abs(host(den)), host(em)) + 1e-6)[:, :, None]); pos += n
    return np.concatenate(got), mem


@pytest.mark.parametrize("H,D,V", [(2, 1, 1), (3, 7, 5), (2, 8, 8), (1, 16, 3), (3, 17, 16), (2, 32, 31), (4, 33, 2), (2, 64, 32), (1, 100, 140), (1, 127, 9), (2, 128, 64), (1, 200, 20),
                                   (1, 255, 33), (1, 256, 40), (1, 300, 12), (1, 400, 7), (1, 512, 16), (1, 511, 3)])
def test_matrix_memory_and_state_hand_over(H, D, V):
    rng = np.random.default_rng(H * 1000 + D)
    T, cap = 37, 6.0
    x = memory_inputs(rng, T, H, D, V)
    ref, (S, n, m) = memory_ref(*x, cap)
    for sizes, ld in (([T], None), ([1] * T, 128), ([2, 16, 1, 15, 3], 2 * H + 1)):
        got, mem = run_memory(x, cap, sizes, rng, ld=ld)
        np.testing.assert_allclose(got, ref, rtol=3e-4, atol=3e-5 * np.abs(ref).max())
        np.testing.assert_allclose(host(mem.m), m, rtol=1e-5, atol=1e-5)
        st = host(mem.state)
        np.testing.assert_allclose(st[:, :V].transpose(0, 2, 1), S, rtol=3e-4, atol=3e-5 * max(np.abs(S).max(), 1e-3))
        np.testing.assert_allclose(st[:, V], n, rtol=3e-4, atol=3e-5 * max(np.abs(n).max(), 1e-3))


@pytest.mark.parametrize("bias,cap", [((-8.0, 6.0), 15.0), ((9.0, -3.0), 15.0), ((0.0, 0.0), 0.5), ((-14.0, -12.0), 12.0), ((14.0, 14.0), 12.0)])
def test_gates_far_from_balance(bias, cap):
    """Tiny input gates (the quotient is e^-m), huge ones, a low cap, everything forgotten, everything kept."""
    rng = np.random.default_rng(int(cap * 10))
    T, H, D, V = 90, 2, 12, 9
    x = memory_inputs(rng, T, H, D, V, bias, 1.0)
    ref, _ = memory_ref(*x, cap)
    for sizes in ([T], [1] * T, [3, 50, 37]):
        got, _ = run_memory(x, cap, sizes, rng)
        np.testing.assert_allclose(got, ref, rtol=1e-3, atol=1e-4 * np.abs(ref).max())


@pytest.mark.parametrize("H,D,V", [(2, 5, 7), (1, 16, 40), (3, 64, 64), (2, 33, 5), (2, 128, 31), (1, 256, 30), (2, 20, 20), (1, 300, 10)])
def test_memory_segments_side_by_side(H, D, V):
    """Long steps run as segments whose states are joined; steps that start later, that end inside a tile or a segment, and short ones between."""
    rng = np.random.default_rng(D)
    T, cap = 1100, 10.0
    x = memory_inputs(rng, T, H, D, V, (-1.0, 5.0))                           # slow decays: states cross many segments
    ref, _ = memory_ref(*x, cap)
    for sizes in ([T], [5, 1000, 95], [517, 583], [1024, 1, 75]):
        got, _ = run_memory(x, cap, sizes, rng, segments=True)
        np.testing.assert_allclose(got, ref, rtol=1e-3, atol=2e-4 * np.abs(ref).max())


def test_memory_keeps_a_far_write_under_an_open_forget_gate_and_loses_it_under_a_closed_one():
    rng = np.random.default_rng(5)
    T, H, D, V, cap = 700, 2, 8, 6, 15.0
    for fb, alive in ((9.0, True), (0.0, False)):
        q, k, v, zi, zf, bi, bf = memory_inputs(rng, T, H, D, V, (-3.0, fb), 0.1)
        zi[3], k[3], q = 12.0, 3.0, np.abs(q)                                 # one write stands out, and every query finds it
        x = (q, k, v, zi, zf, bi, bf)
        ref, _ = memory_ref(*x, cap)
        v2 = v.copy(); v2[3] += 5.0
        moved = np.abs(memory_ref(q, k, v2, zi, zf, bi, bf, cap)[0][-1] - ref[-1]).max()
        assert (moved > 1.0) == alive
        for sizes in ([T], [4, 696], [600] + [1] * 100):
            got, _ = run_memory(x, cap, sizes, rng, segments=True)
            np.testing.assert_allclose(got, ref, rtol=1e-3, atol=2e-4 * np.abs(ref).max())


@pytest.mark.parametrize("H,D,V", [(2, 1, 1), (3, 9, 11), (2, 20, 16), (2, 64, 64), (1, 128, 200), (2, 36, 70), (1, 256, 520), (1, 250, 40), (1, 512, 256), (30, 32, 64), (1, 4, 3)])
def test_memory_token_equals_the_rows(H, D, V):
    """The one-launch token form: gates, memory, head norm over the cluster, output gate; and the rows' own last step."""
    rng = np.random.default_rng(D * 10 + V)
    T, eps, n, cap = 9, 1e-4, H * V, 7.0
    x = memory_inputs(rng, T, H, D, V)
    q, k, v, zi, zf, bi, bf = x
    gate, norm = rng.standard_normal((T, n)), 1 + 0.3 * rng.standard_normal(n)
    ref = O.rms(memory_ref(*x, cap)[0], eps).reshape(T, n) * norm * O.sigmoid(gate)
    mem = Memory(rng, H, D, V)
    for t in range(T):
        out = torch.empty(n, device="cuda")
        lib().nt_b200_mlstm_token(out.data_ptr(), dp(q[t]), dp(k[t]), dp(v[t]), dp(gate[t]), dp(zi[t]), dp(zf[t]), dp(bi), dp(bf), dp(norm), mem.state.data_ptr(), mem.m.data_ptr(), cap,
                                  D ** -0.5, eps, H, D, V, t, stream())
        np.testing.assert_allclose(host(out), ref[t], rtol=1e-3, atol=1e-3)
    mem = Memory(rng, H, D, V)
    o, den, em = mem.rows(q[:5], k[:5], v[:5], zi[:5], zf[:5], bi, bf, cap, 0)   # rows first, then tokens from the state they left
    out, sp = torch.empty(5, n, device="cuda"), split_buffer(5, n)
    lib().nt_b200_mlstm_out_norm(out.data_ptr(), sp.data_ptr(), o.data_ptr(), den.data_ptr(), em.data_ptr(), dp(gate[:5]), dp(norm), eps, 5, H, V, stream())
    np.testing.assert_allclose(host(out), ref[:5], rtol=1e-3, atol=1e-3)
    np.testing.assert_allclose(joined(sp, 5, n), ref[:5], rtol=1e-3, atol=1e-3)
    for t in range(5, T):
        out = torch.empty(n, device="cuda")
        lib().nt_b200_mlstm_token(out.data_ptr(), dp(q[t]), dp(k[t]), dp(v[t]), dp(gate[t]), dp(zi[t]), dp(zf[t]), dp(bi), dp(bf), dp(norm), mem.state.data_ptr(), mem.m.data_ptr(), cap,
                                  D ** -0.5, eps, H, D, V, t, stream())
        np.testing.assert_allclose(host(out), ref[t], rtol=1e-3, atol=1e-3)


# ---------------------------------------------------------------- router
@pytest.mark.parametrize("E,top,groups", [(5, 2, None), (1, 1, None), (8, 4, (4, 3)), (6, 2, (3, 1)), (6, 2, (3, 2)), (33, 33, None), (256, 8, (8, 3)), (256, 4, (256, 9)), (64, 3, (1, 1)),
                                          (64, 64, (2, 2)), (96, 5, (48, 40)), (40, 2, (2, 1))])
def test_router_shares_inside_the_best_groups(E, top, groups):
    rng = np.random.default_rng(E)
    T, W = 11, 52
    h, R = rng.standard_normal((T, W)), rng.standard_normal((E, W)) * 0.4
    g = {"count": groups[0], "keep": groups[1]} if groups else None
    gc, gk = groups or (0, 0)
    sel_ref, wt_ref = O.route(h, R, top, g)
    sel, wt = torch.zeros(T, top, device="cuda", dtype=torch.int32), torch.zeros(T, top, device="cuda")
    lib().nt_b200_moe_route_shares(sel.data_ptr(), wt.data_ptr(), dp(h), dp(R), E, top, gc, gk, W, T, stream())
    np.testing.assert_array_equal(sel.cpu().numpy(), sel_ref)
    np.testing.assert_allclose(host(wt), wt_ref, rtol=5e-5, atol=1e-7)
    np.testing.assert_allclose(host(wt).sum(1), 1.0, rtol=1e-5)
    if groups and gk < min(gc, top):                                          # `top` groups or more always hold the best experts
        assert (sel_ref != O.route(h, R, top)[0]).any()
    # equal logits: the lowest groups and indices are chosen
    lib().nt_b200_moe_route_shares(sel.data_ptr(), wt.data_ptr(), dp(np.zeros((T, W))), dp(R), E, top, gc, gk, W, T, stream())
    np.testing.assert_array_equal(sel.cpu().numpy(), np.tile(np.arange(top), (T, 1)))
    np.testing.assert_allclose(host(wt), 1.0 / top, rtol=1e-5)
    # the decode step's choice, made by the expert kernel from the logits
    ff = 3
    Gs, Us = O.bf16_grid(rng.standard_normal((E, ff, W))), O.bf16_grid(rng.standard_normal((E, ff, W)))
    gd, ud = dev(Gs), dev(Us)
    tab = lambda t: torch.tensor([t[e].data_ptr() for e in range(E)], device="cuda", dtype=torch.int64)
    gt, ut = tab(gd), tab(ud)
    for t in (0, T - 1):
        act = torch.zeros(top * ff, device="cuda")
        lib().nt_b200_moe_choose_up_shares(act.data_ptr(), sel.data_ptr(), wt.data_ptr(), dp(h[t]), dp(R @ h[t]), gt.data_ptr(), ut.data_ptr(), int(DType.F32), E, top, gc, gk, ff, W,
                                           stream())
        np.testing.assert_array_equal(sel.cpu().numpy()[0], sel_ref[t])
        np.testing.assert_allclose(host(wt)[0], wt_ref[t], rtol=5e-5, atol=1e-7)
        np.testing.assert_allclose(host(act), np.concatenate([O.silu(Gs[e] @ h[t]) * (Us[e] @ h[t]) for e in sel_ref[t]]), rtol=1e-4, atol=1e-4)


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


AT, LA, ML = "attention", "latent_attention", "mlstm"
CONFIGS = {
    "base": dict(),
    "borrowed_rows": dict(pattern=(ML, AT, LA, AT, AT), mlp=("moe", "dense", None), kv_from={3: 1, 4: 1}),
    "memory_first_other_feed_forwards": dict(pattern=(ML, ML, LA), mlp=("dense", None, "moe"), groups=None, scaling=None),
    "memory_only": dict(pattern=(ML, ML, ML), mlp=("moe", None, "dense"), shared=0, m_heads=4, m_dim=16, m_vdim=16),
    "plain_attention_top_of_all": dict(pattern=(AT, LA), mlp=("moe",), temp=None, experts=4, top=4, groups=(4, 4), heads=4, kv_heads=4, dim=8, vdim=8),
    "one_layer_one_expert": dict(pattern=(LA,), mlp=("moe",), experts=3, top=1, groups=(1, 1), shared=12, eff=12, rot_dim=2),
    "every_size_one": dict(pattern=(ML, LA, AT), mlp=("dense", "moe"), width=1, vocab=5, heads=1, kv_heads=1, dim=1, vdim=1, temp=(1.0, 1), l_heads=1, l_dim=1, rot_dim=2, l_vdim=1, q_rank=1,
                           kv_rank=1, m_heads=1, m_dim=1, m_vdim=1, cap=1.0, ff=1, experts=1, top=1, groups=(1, 1), eff=1, shared=1),
    "unrotated_wide_latent": dict(pattern=(LA, ML), mlp=("dense", "moe"), rot_dims=0, rot_dim=4, l_dim=12, kv_rank=300, l_vdim=20, l_heads=5, groups=(2, 1), top=3),
    "heads_wider_than_the_tiled_kernel": dict(pattern=(LA, AT, ML), mlp=(None, "dense"), l_dim=180, rot_dim=20, l_vdim=130, l_heads=2, heads=2, kv_heads=1, dim=140, vdim=260, m_dim=40,
                                              m_vdim=150),
    "partly_rotated": dict(pattern=(LA,), mlp=(None,), rot_dim=10, rot_dims=4, scaling=(3.0, 30, 6.0, 0.5)),
    # tile-aligned matrices: with BF16 weights the projections run on the tensor cores, short ones through padded copies, the attention on the tiled kernel
    "tensor_core_tiles": dict(width=128, vocab=128, heads=2, kv_heads=1, dim=64, vdim=64, l_heads=2, l_dim=40, rot_dim=24, l_vdim=48, q_rank=64, kv_rank=64, m_heads=4, m_dim=32, m_vdim=48,
                              ff=192, experts=4, top=2, groups=(2, 1), eff=128, shared=128),
    "tensor_core_tiles_ragged": dict(width=192, vocab=100, heads=6, kv_heads=2, dim=96, vdim=96, l_heads=3, l_dim=64, rot_dim=32, l_vdim=80, q_rank=192, kv_rank=96, m_heads=3, m_dim=64,
                                     m_vdim=64, ff=320, experts=6, top=3, groups=(3, 2), eff=64, shared=192),
    "wide_projections_in_one_launch": dict(pattern=(ML, LA, AT, ML), mlp=("moe",), width=128, vocab=90, heads=8, kv_heads=4, dim=64, vdim=128, l_heads=8, l_dim=32, rot_dim=32, l_vdim=64,
                                           q_rank=256, kv_rank=224, m_heads=4, m_dim=64, m_vdim=96, experts=8, top=3, groups=(4, 2), eff=128, shared=256),
    "sixty_four_gate_rows": dict(pattern=(ML, AT), mlp=("dense",), width=128, m_heads=64, m_dim=4, m_vdim=4, heads=8, kv_heads=2, dim=64, vdim=128, ff=128),
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
    # 16-bit mode: the cache rows are BF16, and the per-head keys and values that prompt portions of 16 rows or more expand latent rows to; everything
    # else is F32 there too, so against an oracle that rounds the same numbers only a few roundings that fall on the other side are left
    ref_dec, ref_pre = (ref, ref) if exact else (O.forward(cfg, W, toks, O.bf16_grid), O.forward(cfg, W, toks, O.bf16_grid, CONFIGS[name].get("l_dim", 9) <= 160))
    tol = 3e-4 if exact else 2e-2
    if cfg["width"] == 1:
        tol = 2e-2 if exact else 2e-1                                    # the norm of one channel is a sign: next to 0 it magnifies rounding
    mixed_tol = tol if exact else tol + 2 * max(rel_rms(ref_dec, ref), rel_rms(ref_pre, ref))      # some portions expand, some do not
    whole = run_portions(m, toks, [S])
    assert rel_rms(whole, ref_pre) < tol
    single = run_portions(m, toks, [1] * S)
    assert rel_rms(single, ref_dec) < tol
    mixed = run_portions(m, toks, [2, 17, 3, 2, 20, 5, 1, 1, 8, 2])      # portions cut anywhere
    assert rel_rms(mixed, ref) < mixed_tol
    assert rel_rms(run_portions(m, toks, [40] + [1] * 21), ref) < mixed_tol
    m.set_prefill_min_tokens(2)                                          # the short portions as prompt rows instead of decode steps
    assert rel_rms(run_portions(m, toks, [2, 17, 3, 2, 20, 5, 1, 1, 8, 2]), ref) < mixed_tol
    if exact and cfg["width"] > 1:                                       # how a prompt is cut changes rounding only
        assert rel_rms(single, whole) < 1e-4 and rel_rms(mixed, whole) < 1e-4
    m.close()


def test_each_mechanism_in_a_model_of_its_own():
    """Models of one layer each, so that a fault names its mechanism."""
    for k, kw in enumerate((dict(pattern=(AT,), mlp=(None,)), dict(pattern=(LA,), mlp=(None,)), dict(pattern=(ML,), mlp=(None,)), dict(pattern=(ML,), mlp=("dense",)),
                            dict(pattern=(ML,), mlp=("moe",)), dict(pattern=(ML,), mlp=("moe",), shared=0), dict(pattern=(ML,), mlp=("moe",), groups=None),
                            dict(pattern=(AT, AT), mlp=(None,), kv_from={1: 0}))):
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
    m.set_prefill_min_tokens(2)
    assert rel_rms(run_portions(m, toks, [2, 3]), ref) < 2e-4
    assert rel_rms(run_portions(m, toks, [2, 1, 2]), ref) < 2e-4
    m.close()


def test_rows_and_states_are_reused_between_requests():
    """A second request starts at position 0 over the first one's cache rows, matrix memories, normalizers and stabilizers: bit-equal to running alone."""
    rng = np.random.default_rng(21)
    cfg, W = O.random_model(rng, kv_from={3: 0})
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


def test_unequal_requests_one_after_the_other_equal_each_alone():
    rng = np.random.default_rng(31)
    cfg, W = O.random_model(rng)
    reqs = [rng.integers(0, cfg["vocab"], n).astype(np.int32) for n in (47, 1, 20, 2, 33)]
    m = build(cfg, W, True)
    for r in reqs + reqs[::-1]:
        assert rel_rms(run_portions(m, r, [len(r)]), O.forward(cfg, W, r)) < 2e-4
    m.close()


def test_prompt_longer_than_one_portion_of_the_engine():
    """2100 tokens: the engine cuts the prompt at 2048, so every state crosses that cut; 2049: the second part is a single row; tile-aligned sizes, both
    modes."""
    rng = np.random.default_rng(3)
    cfg, W = O.random_model(rng, **CONFIGS["tensor_core_tiles"])
    S = 2100
    toks = rng.integers(0, cfg["vocab"], S).astype(np.int32)
    want = [0, 1, 63, 64, 2047, 2048, 2049, S - 1]
    for exact in (True, False):
        ref = O.forward(cfg, W, toks) if exact else O.forward(cfg, W, toks, O.bf16_grid, True)
        m = build(cfg, W, exact, max_context=2304)
        tol = 5e-4 if exact else 2e-2
        assert rel_rms(m.forward_logits(toks, 0, want), ref[want]) < tol
        assert rel_rms(m.forward_logits(toks[:2049], 0, want[:6]), ref[want[:6]]) < tol
        assert rel_rms(m.forward_logits(toks[2049:], 2049, [0, S - 2050]), ref[[2049, S - 1]]) < tol
        m.close()


def test_long_decode_and_graph_replay():
    rng = np.random.default_rng(8)
    cfg, W = O.random_model(rng, pattern=(ML, AT, LA), mlp=("dense", "moe"), width=32, vocab=50, temp=(0.5, 16))
    S = 300
    toks = rng.integers(0, cfg["vocab"], S).astype(np.int32)
    ref = O.forward(cfg, W, toks)
    m = build(cfg, W, True, max_context=512)
    assert rel_rms(run_portions(m, toks, [3] + [1] * (S - 3)), ref) < 3e-4
    m.use_graph(False)
    m.clear_kv()
    assert rel_rms(run_portions(m, toks, [3] + [1] * (S - 3)), ref) < 3e-4
    m.close()


@pytest.mark.parametrize("kind", [AT, LA, ML])
def test_a_far_token_reaches_as_far_as_its_mechanism_lets_it(kind):
    """One layer, so the mixer is the only path between positions.  One token shouts: through attention and through a memory that forgets slowly it must be
    heard hundreds of tokens on, by the oracle's amount, whatever step kinds meet on the way."""
    rng = np.random.default_rng(13)
    S = 420
    cfg, W = O.random_model(rng, pattern=(kind,), mlp=(None,), scale=3.0, l_scale=2.0, heads=3, kv_heads=3, temp=(0.5, 100))
    W["embed"][0] *= 8.0
    if kind == ML:
        W["l0.mix.f.b"][:] = 12.0
        W["l0.mix.f"][:] *= 0.1
    toks = rng.integers(1, cfg["vocab"], S).astype(np.int32)
    base = O.forward(cfg, W, toks)
    m = build(cfg, W, True, max_context=512)
    for at in (0, 5, 16, 64):
        t = toks.copy(); t[at] = 0
        ref = O.forward(cfg, W, t)
        moved = np.sqrt(((ref - base) ** 2).mean(1))
        assert moved[at] > 1e-2 and moved[-40:].max() > 1e-3 and not moved[:at].any()
        for sizes in ([S], [at + 199] + [1] * 3 + [S - at - 202], [3, 300] + [1] * (S - 303)):
            assert rel_rms(run_portions(m, t, sizes), ref) < 3e-4
    m.close()


def test_greedy_generation_through_the_engine(tmp_path):
    rng = np.random.default_rng(4)
    cfg, W = O.random_model(rng, kv_from={3: 0})
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
