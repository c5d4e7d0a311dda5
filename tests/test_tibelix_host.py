"""CPU tests of the Tibelix family: the oracle's own invariants, and the engine's reading of a model folder (what it accepts, what it
refuses and why).  Nothing here needs a GPU: nt_model_dir_describe parses config.json and the safetensors header only."""
import ctypes as C
import math

import numpy as np
import pytest

import tibelix_oracle as O
from zelunex_util import write_model_dir

from ntransformer_b200._lib import lib


def describe(path):
    buf = C.create_string_buffer(1 << 16)
    rc = lib().nt_model_dir_describe(str(path).encode(), buf, len(buf))
    return rc, buf.value.decode()


def test_oracle_is_causal_and_cut_free():
    rng = np.random.default_rng(0)
    cfg, W = O.random_model(rng, kv_from={3: 0})
    toks = rng.integers(0, cfg["vocab"], 40)
    full = O.forward(cfg, W, toks)
    np.testing.assert_allclose(O.forward(cfg, W, toks[:17]), full[:17], rtol=1e-9, atol=1e-9)      # a prefix does not see what follows
    other = toks.copy(); other[30] = (other[30] + 1) % cfg["vocab"]
    np.testing.assert_allclose(O.forward(cfg, W, other)[:30], full[:30], rtol=1e-9, atol=1e-9)


def test_oracle_attention_conventions():
    # slopes halve 8 / H times per head; the temperature steps when position + 1 reaches a multiple of `every`
    np.testing.assert_allclose(O.slopes(8), 2.0 ** -np.arange(1, 9))
    np.testing.assert_allclose(O.slopes(4), [0.25, 0.0625, 2.0 ** -6, 2.0 ** -8])
    t = O.query_temperature([0, 3, 4, 8, 9, 13, 14], 0.5, 5)
    np.testing.assert_allclose(t, [1, 1, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3), 1 + 0.5 * math.log(3), 1 + 0.5 * math.log(4)])
    # the sink takes 1 / (1 + sum): a single key of score 0 gets one half, very low scores leave nothing
    np.testing.assert_allclose(O.sink_softmax(np.array([[0.0]]), np.ones((1, 1), bool)), [[0.5]])
    np.testing.assert_allclose(O.sink_softmax(np.array([[-50.0, -60.0]]), np.ones((1, 2), bool)), np.exp([[-50.0, -60.0]]), rtol=1e-12)
    # equal keys: the bias ranks them by distance, and taking slope * j off instead of slope * (i - j) would not be the same beside a sink
    q, k = np.zeros((3, 1, 2)), np.zeros((3, 1, 2))
    v = np.eye(3).reshape(3, 1, 3)
    o = O.biased_attention(q, k, v, 1.0, np.array([1.0]))
    e = np.exp([-2.0, -1.0, 0.0])
    np.testing.assert_allclose(o[2, 0], e / (1 + e.sum()))


def test_oracle_rotation_conventions():
    # channel 2i turns with 2i + 1, the pair's angle is pos * base^(-2i / dims); the rest pass
    v = np.array([[[1.0, 0.0, 0.0, 1.0, 7.0]]])
    np.testing.assert_allclose(O.rotate_pairs(v, [3], {"dims": 4, "base": 100.0})[0, 0], [np.cos(3.0), np.sin(3.0), -np.sin(0.3), np.cos(0.3), 7.0], atol=1e-12)
    f, mag = O.blended_frequencies(16, 1000.0, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
    plain = 1000.0 ** (-2.0 * np.arange(8) / 16)
    assert mag == pytest.approx(0.1 * math.log(4.0) + 1)
    assert f[0] == plain[0] and f[-1] == pytest.approx(plain[-1] / 4.0)                  # short wavelengths are left, long ones slowed
    assert np.all(f <= plain) and np.all(f >= plain / 4.0 - 1e-15)
    assert np.any((f < plain * 0.999) & (f > plain / 4.0 * 1.001))                       # a ramp between


def test_oracle_matrix_memory_conventions():
    one = np.ones((3, 1, 1))
    # f = 0 (nothing is forgotten), i = 0: m stays 0, S sums k v, the quotient is max(|n q|, 1)
    o, (S, n, m) = O.mlstm_memory(one, one, np.array([2.0, 4.0, 9.0]).reshape(3, 1, 1), np.zeros((3, 1)), np.zeros((3, 1)))
    np.testing.assert_allclose(o[:, 0, 0], [2.0, 3.0, 5.0], rtol=2e-6)
    assert S[0, 0, 0] == 15.0 and n[0, 0] == 3.0 and m[0] == 0.0
    # a large input gate moves the stabilizer, the result is that of the unscaled sums
    i, f = np.array([[3.0], [-1.0], [2.0]]), np.array([[-0.1], [-0.7], [-2.0]])
    v = np.array([2.0, 4.0, 9.0])
    o, (_, _, m) = O.mlstm_memory(one, one, v.reshape(3, 1, 1), i, f)
    s = nn = 0.0
    for t in range(3):
        s, nn = np.exp(f[t, 0]) * s + np.exp(i[t, 0]) * v[t], np.exp(f[t, 0]) * nn + np.exp(i[t, 0])
        np.testing.assert_allclose(o[t, 0, 0], s / max(nn, 1.0), rtol=3e-6)
    assert m[0] == pytest.approx(2.0)                                                   # 3.0 - 0.7 - 2.0 < 2.0
    # the stabilizer starts at 0: a small first input gate leaves it at the forget gate, not at the input gate
    assert O.mlstm_memory(one[:1], one[:1], one[:1], np.array([[-6.0]]), np.array([[-1.0]]))[1][2][0] == -1.0
    np.testing.assert_allclose(O.soft_cap(np.array([0.1, 500.0, -500.0]), 5.0), [5 * np.tanh(0.02), 5.0, -5.0])
    np.testing.assert_allclose(O.log_sigmoid(np.array([0.0, 40.0, -40.0])), [-math.log(2), -math.exp(-40), -40.0], rtol=1e-6)


def test_oracle_router_conventions():
    z = np.array([[1.0, 5.0, 4.0, 4.5, 2.0, 0.0]])
    R = z.T
    sel, wt = O.route(np.ones((1, 1)), R, 2)
    assert sel.tolist() == [[1, 3]]
    np.testing.assert_allclose(wt.sum(), 1.0)
    np.testing.assert_allclose(wt[0, 0] / wt[0, 1], math.exp(0.5))
    # three groups of two, one kept: the one that holds the largest score, although another has the larger sum
    sel, wt = O.route(np.ones((1, 1)), R, 2, {"count": 3, "keep": 1})
    assert sel.tolist() == [[1, 0]]
    np.testing.assert_allclose(wt[0, 0] / wt[0, 1], math.exp(4.0))


def test_frequency_table_matches_the_oracle():
    for dims, base, sc in ((16, 1000.0, (4.0, 64, 8.0, 1.0)), (6, 500.0, (4.0, 40, 8.0, 1.0)), (64, 250000.5, (3.7, 1000, 30.5, 0.9)), (2, 10.0, (2.0, 16, 4.0, 1.0)), (32, 7.0, None)):
        s = dict(zip(("factor", "original", "fast", "slow"), sc)) if sc else None
        want, mag = O.blended_frequencies(dims, base, s)
        got = np.zeros(dims // 2)
        m = lib().nt_b200_rotary_table64(got.ctypes.data_as(C.c_void_p), dims, base, *(sc or (0.0, 0.0, 0.0, 0.0)))
        np.testing.assert_allclose(got, want, rtol=1e-12)
        assert m == pytest.approx(mag, rel=1e-6)


def test_model_folder_is_read_as_configured(tmp_path):
    rng = np.random.default_rng(1)
    cfg, W = O.random_model(rng, kv_from={3: 0})
    rc, text = describe(write_model_dir(tmp_path / "ok", cfg, W))
    assert rc == 0, text
    assert "architecture=Tibelix" in text and "layers=4" in text
    assert "layer 0: heads=6 kv=3 dim=10 vdim=7 window=0 keep=0 ff=23" in text and "mixer=attention temp=0.700000/5.000000 kv_from=-1 bias=1 unit_sink=1 ff_kind=dense" in text
    assert "layer 1: heads=3 kv=1 dim=9 vdim=5 window=0 keep=0 ff=12" in text
    assert "mixer=latent q_rank=13 kv_rank=11 rot_dim=6 rot=6 factor=4.000000 ff_kind=moe experts=6 top=2 route_groups=3/2 shared_ff=17" in text
    assert "layer 2: heads=2 kv=2 dim=9 vdim=11 window=0 keep=0 ff=0" in text and "mixer=mlstm cap=8.000000 ff_kind=none" in text
    assert "kv_from=0" in text and "tensors=%d" % len(W) in text


def test_optional_parts_may_be_absent(tmp_path):
    rng = np.random.default_rng(3)
    cfg, W = O.random_model(rng, mlp=(None, "moe"), shared=0, groups=None, scaling=None, temp=None)
    cfg["layers"][1]["mixer"].pop("rot")
    rc, text = describe(write_model_dir(tmp_path / "ok", cfg, W))
    assert rc == 0, text
    assert "ff_kind=none" in text and "shared_ff=0" in text and "route_groups=0/0" in text and "temp=0.000000/0.000000" in text and "rot=0 factor=0" in text
    assert "tensors=%d" % len(W) in text


@pytest.mark.parametrize("what", ["missing_tensor", "missing_inner_norm", "wrong_shape", "odd_rot", "rot_over_dim", "unknown_mixer", "unknown_ff", "top_over_experts", "missing_key",
                                  "heads_do_not_divide", "zero_cap", "groups_do_not_divide", "kept_groups_too_small", "kv_from_later", "kv_from_another_mixer", "kv_from_a_borrower",
                                  "kv_from_other_heads", "gate_rows_for_channels", "temperature_without_step", "scaling_incomplete"])
def test_bad_model_folders_are_refused(tmp_path, what):
    rng = np.random.default_rng(2)
    cfg, W = O.random_model(rng, pattern=("attention", "latent_attention", "mlstm", "attention", "attention"), kv_from={4: 0})
    L = cfg["layers"]
    if what == "missing_tensor":
        del W["l2.mix.f.b"]
    elif what == "missing_inner_norm":
        del W["l1.norm2b"]
    elif what == "wrong_shape":
        W["l1.mix.uk"] = W["l1.mix.uk"][:, :3]
    elif what == "odd_rot":
        L[1]["mixer"]["rot"]["dims"] = 3
    elif what == "rot_over_dim":
        L[1]["mixer"]["rot"]["dims"] = 8
    elif what == "unknown_mixer":
        L[2]["type"] = "convolution"
    elif what == "unknown_ff":
        L[0]["mlp"]["kind"] = "gated"
    elif what == "top_over_experts":
        L[1]["mlp"]["router"]["top"] = 7
    elif what == "missing_key":
        del L[0]["mixer"]["scale"]
    elif what == "heads_do_not_divide":
        L[0]["mixer"]["kv_heads"] = 4
    elif what == "zero_cap":
        L[2]["mixer"]["gate_cap"] = 0
    elif what == "groups_do_not_divide":
        L[1]["mlp"]["router"]["groups"]["count"] = 4
    elif what == "kept_groups_too_small":
        L[1]["mlp"]["router"].update(top=3, groups={"count": 3, "keep": 1})
    elif what == "kv_from_later":
        L[3]["mixer"]["kv_from"] = 4
    elif what == "kv_from_another_mixer":
        L[4]["mixer"]["kv_from"] = 1
    elif what == "kv_from_a_borrower":
        L[3]["mixer"]["kv_from"] = 0
        L[4]["mixer"]["kv_from"] = 3
    elif what == "kv_from_other_heads":
        L[4]["mixer"]["kv_heads"] = 2
    elif what == "gate_rows_for_channels":
        W["l2.mix.g"] = W["l2.mix.g"][:2]
    elif what == "temperature_without_step":
        L[0]["mixer"]["q_temp"]["every"] = 0
    elif what == "scaling_incomplete":
        del L[1]["mixer"]["rot"]["scaling"]["slow"]
    rc, text = describe(write_model_dir(tmp_path / what, cfg, W))
    assert rc != 0, text
