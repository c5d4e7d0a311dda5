"""CPU tests of the Fuvozen family: the oracle's own invariants, and the engine's reading of a model folder (what it accepts, what it
refuses and why).  Nothing here needs a GPU: nt_model_dir_describe parses config.json and the safetensors header only."""
import ctypes as C

import numpy as np
import pytest

import fuvozen_oracle as O
from zelunex_util import write_model_dir

from ntransformer_b200._lib import lib


def describe(path):
    buf = C.create_string_buffer(1 << 16)
    rc = lib().nt_model_dir_describe(str(path).encode(), buf, len(buf))
    return rc, buf.value.decode()


def test_oracle_is_causal_and_cut_free():
    rng = np.random.default_rng(0)
    cfg, W = O.random_model(rng)
    toks = rng.integers(0, cfg["vocab"], 40)
    full = O.forward(cfg, W, toks)
    np.testing.assert_allclose(O.forward(cfg, W, toks[:17]), full[:17], rtol=1e-9, atol=1e-9)      # a prefix does not see what follows
    other = toks.copy(); other[30] = (other[30] + 1) % cfg["vocab"]
    np.testing.assert_allclose(O.forward(cfg, W, other)[:30], full[:30], rtol=1e-9, atol=1e-9)


def test_oracle_conventions():
    # pair hashing: the first token reads the row behind the buckets
    assert list(O.bigram_rows([5, 9, 2], 10, 3, 7)) == [10, (15 + 63) % 10, (27 + 14) % 10]
    # channel 2i turns with 2i + 1, the pair's angle is pos * base^(-2i / dims); the rest pass
    v = np.array([[[1.0, 0.0, 0.0, 1.0, 7.0]]])
    np.testing.assert_allclose(O.rotate_pairs(v, [3], 4, 100.0)[0, 0], [np.cos(3.0), np.sin(3.0), -np.sin(0.3), np.cos(0.3), 7.0], atol=1e-12)
    assert O.window_mask(5, 2).sum(1).tolist() == [1, 2, 2, 2, 2] and O.window_mask(5, None).sum() == 15
    # grouped norm: every run has root mean square 1
    n = O.norm_groups(np.array([[3.0, 3.0, 0.1, -0.1]]), np.ones(4), 2, 0.0)
    np.testing.assert_allclose(n, [[1.0, 1.0, 1.0, -1.0]])
    # the read-out sees the current token through the bonus only, later tokens see it through the state (decayed once per later step)
    one = np.ones((3, 1, 1))
    o = O.wkv_recurrence(one, one, np.array([2.0, 0.0, 0.0]).reshape(3, 1, 1), 0.5 * one, np.array([[3.0]]))
    np.testing.assert_allclose(o[:, 0, 0], [6.0, 2.0, 1.0])
    # shares over ALL experts, not renormalized over the chosen
    sel, wt = O.route(np.ones((1, 1)), np.log(np.array([[1.0], [2.0], [5.0]])), 2, 3.0)
    assert sel.tolist() == [[2, 1]]
    np.testing.assert_allclose(wt, [[3.0 * 5 / 8, 3.0 * 2 / 8]])
    # both branches of the activation meet at 0 with slope 1/2
    z = np.array([-1e-6, 0.0, 1e-6])
    np.testing.assert_allclose(O.xielu(z, 0.3, -0.4), 0.5 * z, atol=1e-11)
    np.testing.assert_allclose(O.xielu(np.array([2.0, -1.0]), 0.0, 0.0), [4 * np.log(2) + 1, (0.5 + np.log(2)) * np.exp(-1.0) - 0.5])


def test_model_folder_is_read_as_configured(tmp_path):
    rng = np.random.default_rng(1)
    cfg, W = O.random_model(rng)
    for L in cfg["layers"]:
        if L["type"] == "wkv":
            del L["mixer"]["decay_rank"]                                                              # read from the tensor's shape
    rc, text = describe(write_model_dir(tmp_path / "ok", cfg, W))
    assert rc == 0, text
    assert "architecture=Fuvozen" in text and "layers=4" in text
    assert "layer 0: heads=2 kv=2 dim=9 vdim=9 window=0 keep=0 ff=23" in text and "mixer=wkv decay_rank=5 ff_kind=dense" in text
    assert "layer 1: heads=3 kv=1 dim=10 vdim=7 window=9 keep=0 ff=12" in text
    assert "mixer=latent kv_rank=11 rot_dim=6 rot=6 ff_kind=moe experts=5 top=2 route_scale=1.700000 shared_ff=17 norm_groups=3 buckets=97" in text
    assert "tensors=%d" % len(W) in text


def test_optional_parts_may_be_absent(tmp_path):
    rng = np.random.default_rng(3)
    cfg, W = O.random_model(rng, mlp=(None, "moe"), shared=0, window=0)
    rc, text = describe(write_model_dir(tmp_path / "ok", cfg, W))
    assert rc == 0, text
    assert "ff_kind=none" in text and "shared_ff=0" in text and "tensors=%d" % len(W) in text


@pytest.mark.parametrize("what", ["missing_tensor", "wrong_shape", "odd_rot", "rot_over_dim", "groups_do_not_divide", "unknown_mixer", "unknown_ff", "top_over_experts",
                                  "missing_key", "missing_groups", "rank_tensor_missing", "zero_window", "depth_weights_too_short", "pair_table_too_short"])
def test_bad_model_folders_are_refused(tmp_path, what):
    rng = np.random.default_rng(2)
    cfg, W = O.random_model(rng)
    L = cfg["layers"]
    if what == "missing_tensor":
        del W["l0.mix.mu.g"]
    elif what == "wrong_shape":
        W["l1.mix.uk"] = W["l1.mix.uk"][:, :3]
    elif what == "odd_rot":
        L[1]["mixer"]["rot"]["dims"] = 3
    elif what == "rot_over_dim":
        L[1]["mixer"]["rot"]["dims"] = 8
    elif what == "groups_do_not_divide":
        cfg["norm"]["groups"] = 5
    elif what == "unknown_mixer":
        L[2]["type"] = "convolution"
    elif what == "unknown_ff":
        L[2]["mlp"]["kind"] = "gated"
    elif what == "top_over_experts":
        L[1]["mlp"]["router"]["top"] = 6
    elif what == "missing_key":
        del L[1]["mixer"]["scale"]
    elif what == "missing_groups":
        del cfg["norm"]["groups"]
    elif what == "rank_tensor_missing":
        del L[0]["mixer"]["decay_rank"]
        del W["l0.mix.w1"]
    elif what == "zero_window":
        L[1]["mixer"]["mask"]["size"] = 0
    elif what == "depth_weights_too_short":
        W["l2.dwa"] = W["l2.dwa"][:3]
    elif what == "pair_table_too_short":
        W["bigram"] = W["bigram"][:-1]
    rc, text = describe(write_model_dir(tmp_path / what, cfg, W))
    assert rc != 0, text
