"""Pins the plain Papunex reference (tests/papunex_ref.py) with cases small enough to do by hand, and checks the package's host-side parts
(configuration, tensor inventory, frequency table, stacked pieces) against it.  No GPU."""
import numpy as np
import pytest

from crabml_b200 import models, papunex, rotary
from crabml_b200.capi import TensorError
from crabml_b200.seqmodel import Uploader
from tests import papunex_ref as R
from tests.papunex_common import config, dense, latent, mamba, mixed_config, moe


def test_rms_norm_has_eps_inside_the_root():
    x = np.array([3.0, 4.0])
    assert np.allclose(R.rms_norm(x, np.array([2.0, 1.0]), 2.5), x / np.sqrt(12.5 + 2.5) * [2.0, 1.0])


def test_rotation_pairs_neighbours():
    x = np.zeros((4, 4)); x[3] = [1.0, 2.0, 3.0, 4.0]
    out = R.rotate_neighbours(x, 100.0)[3]
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    assert np.allclose(out, [np.cos(a0) - 2 * np.sin(a0), 2 * np.cos(a0) + np.sin(a0), 3 * np.cos(a1) - 4 * np.sin(a1), 4 * np.cos(a1) + 3 * np.sin(a1)])
    y = np.array([[1.0, 2.0, 3.0, 4.0]])
    assert np.allclose(R.rotate_neighbours(y, 100.0), y)                  # position 0 does not turn


def test_frequency_table_of_the_package_is_the_reference_rule():
    for dims, base in ((2, 10.0), (6, 100.0), (64, 3e6), (40, 2e5)):
        f, mag = rotary.table_of({"dims": dims, "base": base})
        assert mag == 1.0 and f.dtype == np.float32 and np.allclose(f, float(base) ** (-2.0 * np.arange(dims // 2) / dims), rtol=1e-7)
        x = np.zeros((6, dims)); x[5, 0::2] = 1.0
        assert np.allclose(R.rotate_neighbours(x, base)[5, 1::2], np.sin(5 * f.astype(np.float64)), atol=1e-6)


def test_sink_counts_once_has_no_value_and_is_not_scaled():
    assert np.allclose(R.softmax_with_sink(np.zeros(3), np.log(5.0)), [1 / 8.0] * 3)
    assert np.allclose(R.softmax_with_sink(np.array([100.0, 0.0]), -1e30), [1.0, 0.0])
    assert np.abs(R.softmax_with_sink(np.array([1.0, 2.0]), 90.0)).max() < 1e-30


def _identity_attention():
    """one head; queries, gate and output pass the input's first columns on"""
    D = 4
    m = {"heads": 1, "dim": 2, "rot_dim": 2, "vdim": 2, "kv_rank": 2, "scale": 1.0, "rot": {"dims": 2, "base": 10.0}}
    w = {"m.q": np.zeros((4, D)), "m.dkv": np.eye(4, D), "m.dkv.norm": np.ones(2), "m.uk": np.eye(2), "m.uv": np.eye(2), "m.sink": np.array([-1e30]), "m.g": np.zeros((2, D)), "m.o": np.eye(D, 2)}
    return m, w


def test_attention_is_causal_and_the_gate_multiplies_element_by_element():
    m, w = _identity_attention()
    h = np.array([[1.0, 0.0, 0, 0], [0.0, 1.0, 0, 0], [1.0, 1.0, 0, 0]])
    c, r = R.latent_rows(h, w, "m.", m, 1e-9)
    out = R.latent_attention(h, (c, r), w, "m.", m)                       # all scores 0: the mean of the values so far, gated by 1/2
    for i in range(3):
        assert np.allclose(out[i, :2], c[:i + 1].mean(0) / 2)
    w["m.g"] = np.array([[9.0, 0, 0, 0], [0, -9.0, 0, 0]])
    g = R.sigmoid(h @ w["m.g"].T)
    assert np.allclose(R.latent_attention(h, (c, r), w, "m.", m)[2, :2], c.mean(0) * g[2])


def test_the_rotated_key_part_is_not_normed_and_the_latent_is():
    m, w = _identity_attention()
    h = np.array([[3.0, 4.0, 5.0, 6.0]])
    c, r = R.latent_rows(h, w, "m.", m, 0.0)
    assert np.allclose(c, np.array([[3.0, 4.0]]) / np.sqrt(12.5)) and np.allclose(r, [[5.0, 6.0]])


def test_score_scale_covers_both_parts():
    m, w = _identity_attention()
    m["scale"] = 0.5
    w["m.q"] = np.eye(4)
    h = np.array([[1.0, 0.0, 2.0, 0.0], [1.0, 0.0, 3.0, 0.0]])
    c, r = R.latent_rows(h, w, "m.", m, 0.0)
    q = h[1].copy(); q[2:] = R.rotate_neighbours(np.array([[0, 0], q[2:]]), 10.0)[1]
    s = np.array([(q[:2] @ c[j] + q[2:] @ r[j]) * 0.5 for j in range(2)])
    p = np.exp(s) / np.exp(s).sum()
    assert np.allclose(R.latent_attention(h, (c, r), w, "m.", m)[1, :2], (p @ c) * 0.5)


def test_convolution_sees_zeros_before_the_start_and_its_last_tap_is_the_current_token():
    x = np.array([[1.0], [10.0], [100.0]])
    assert np.allclose(R.causal_conv(x, np.array([[3.0, 2.0, 1.0]]), np.array([0.5]))[:, 0], [1.5, 12.5, 123.5])


def test_state_space_two_steps_by_hand():
    x = np.array([[[2.0]], [[3.0]]]); B = np.array([[[1.0, 0.5]], [[0.0, 2.0]]]); C = np.array([[[1.0, 1.0]], [[4.0, 0.25]]])
    dt, a_log, d = np.array([[0.5], [0.25]]), np.array([np.log(2.0)]), np.array([10.0])
    s0 = 0.5 * np.array([1.0, 0.5]) * 2.0
    s1 = np.exp(-2.0 * 0.25) * s0 + 0.25 * np.array([0.0, 2.0]) * 3.0
    assert np.allclose(R.state_space(x, B, C, dt, a_log, d)[:, 0, 0], [s0 @ [1.0, 1.0] + 20.0, s1 @ [4.0, 0.25] + 30.0])


def test_heads_share_groups_as_neighbours():
    rng = np.random.default_rng(0)
    x, B, C = np.ones((1, 4, 1)), rng.standard_normal((1, 2, 3)), rng.standard_normal((1, 2, 3))
    y = R.state_space(x, B, C, np.ones((1, 4)), np.zeros(4), np.zeros(4))[0, :, 0]
    d0, d1 = B[0, 0] @ C[0, 0], B[0, 1] @ C[0, 1]
    assert np.allclose(y, [d0, d0, d1, d1])


def test_gate_comes_before_the_norm_and_groups_have_their_own_root_mean_square():
    y, z = np.array([[1.0, 2.0, 30.0, 40.0]]), np.array([[0.5, -1.0, 2.0, 3.0]])
    g = y * z / (1 + np.exp(-z))
    want = np.concatenate([g[:, :2] / np.sqrt((g[:, :2] ** 2).mean() + 0.1), g[:, 2:] / np.sqrt((g[:, 2:] ** 2).mean() + 0.1)], 1) * [1, 2, 3, 4]
    assert np.allclose(R.gate_then_group_norm(y, z, np.array([1.0, 2, 3, 4]), 2, 0.1), want)


def test_router_weights_sum_to_the_scale_and_the_softmax_runs_over_all_experts():
    ids, wts = R.route(np.array([[1.0]]), np.array([[0.0], [2.0], [1.0], [-5.0]]), 2, 1.5)
    assert ids.tolist() == [[1, 2]] and np.allclose(wts.sum(), 1.5)
    assert np.allclose(wts[0, 0] / wts[0, 1], np.e)


def test_squared_relu_and_the_shared_expert():
    assert np.allclose(R.relu_squared(np.array([-3.0, 0.0, 2.0])), [0.0, 0.0, 4.0])
    h = np.array([[1.0, -1.0]])
    w = {"f.router": np.zeros((2, 2)), "f.shared.up": np.array([[2.0, 0.0]]), "f.shared.down": np.array([[1.0], [3.0]]), "f.shared.sg": np.array([[0.0, 1.0]])}
    for e in range(2):
        w[f"f.e{e}.up"], w[f"f.e{e}.down"] = np.array([[float(e + 1), 0.0]]), np.array([[1.0], [0.0]])
    out = R.mixture(h, w, "f.", {"router": {"experts": 2, "top": 1, "scale": 3.0}, "shared": {"ff": 1}})
    assert np.allclose(out, [[3.0 * 1.0 + 4.0 * R.sigmoid(-1.0), 12.0 * R.sigmoid(-1.0)]])


def test_soft_cap():
    assert np.allclose(R.soft_cap(np.array([0.1, 1e9, -1e9]), 7.0), [7 * np.tanh(0.1 / 7), 7.0, -7.0])


def test_forward_is_causal_and_taps_every_layer():
    conf = mixed_config()
    w = papunex.random_weights(papunex.parse_config(conf), 3)
    a = [5, 9, 2, 44, 1, 0, 17, 30, 30, 8, 3, 21, 40]
    b = a[:7] + [31] + a[8:]
    la, lb = R.forward(conf, w, a), R.forward(conf, w, b)
    assert np.allclose(la[:7], lb[:7]) and np.abs(la[7:] - lb[7:]).max() > 1e-3
    taps = []
    R.forward(conf, w, a, taps)
    assert len(taps) == 6 and taps[0].shape == (len(a), conf["width"])

def test_a_shared_cache_is_the_other_layers():
    # the first layer adds nothing (its W_o is zero), so both layers read the same stream: the second one, reading the first one's cache, is a
    # lone layer with the first one's latent projection
    conf = papunex.parse_config(config([latent(mlp=None), latent(heads=2, dim=4, vdim=5, scale=0.7, kv_from=0, mlp=None)]))
    w = papunex.random_weights(conf, 4)
    w["l0.mix.o"] = np.zeros_like(w["l0.mix.o"])
    lone = papunex.parse_config(config([latent(heads=2, dim=4, vdim=5, scale=0.7, mlp=None)]))
    w1 = {n: w[n.replace("l0.", "l0." if "dkv" in n else "l1.")] for n in papunex.expected_tensors(lone)}
    toks = [3, 9, 1, 50, 9, 9, 20]
    assert np.allclose(R.forward(conf, w, toks), R.forward(lone, w1, toks))


def test_config_defaults_and_refusals():
    c = papunex.parse_config(mixed_config())
    assert papunex.parse_config(c) == c                  # parsing what was parsed changes nothing
    assert c["layers"][0]["mlp"] is None and c["layers"][1]["mixer"]["kv_from"] is None and c["layers"][4]["mixer"]["kv_from"] == 1 and c["layers"][2]["mlp"]["shared"] is None
    bare = config([mamba(), latent()], softcap=0)
    del bare["embedding"]
    del bare["layers"][0]["mixer"]["groups"], bare["layers"][0]["mixer"]["norm_groups"], bare["layers"][0]["mlp"]["router"]["scale"]
    p = papunex.parse_config(bare)
    assert p["embedding"]["scale"] == 1.0 and p["logit_softcap"] == 0.0 and p["layers"][0]["mixer"]["groups"] == 1 and p["layers"][0]["mlp"]["router"]["scale"] == 1.0
    for bad in (config([latent(kv_from=0)]), config([latent(), latent(kv_from=1)]), config([mamba(), latent(kv_from=0)]), config([latent(), latent(kv_from=0), latent(kv_from=1)]),
                config([latent(), latent(kv_from=0, kv_rank=15)]), config([latent(), latent(kv_from=0, rot_dim=4)]), config([latent(), latent(kv_from=0, base=499.0)]),
                config([latent(rot_dim=5)]), config([mamba(heads=5)]), config([mamba(norm_groups=7)]), config([mamba(mlp=moe(top=7))]), config([dict(latent(), type="attention")]),
                config([latent(mlp={"kind": "glu", "ff": 4})]), dict(mixed_config(), architecture="Other")):
        with pytest.raises(TensorError):
            papunex.parse_config(bad)


def test_tensor_inventory_and_registry():
    c = papunex.parse_config(mixed_config())
    t = papunex.expected_tensors(c)
    assert t["l1.mix.q"] == [3 * 14, 36] and t["l1.mix.dkv"] == [20, 36] and t["l1.mix.dkv.norm"] == [14] and t["l1.mix.uk"] == [24, 14] and t["l1.mix.g"] == [30, 36]
    assert "l4.mix.dkv" not in t and "l4.mix.dkv.norm" not in t and t["l4.mix.uk"] == [20, 14] and t["l4.mix.uv"] == [15, 14] and t["l4.mix.sink"] == [5]
    assert "l0.norm2" not in t and t["l3.norm2"] == [36] and t["l3.mix.in"] == [30 + 30 + 42 + 6, 36] and t["l3.mix.conv"] == [72, 5]
    assert t["l4.mlp.shared.up"] == [9, 36] and t["l4.mlp.shared.sg"] == [1, 36] and "l2.mlp.shared.up" not in t and t["l2.mlp.e4.down"] == [36, 16]
    w = papunex.random_weights(c, 0)
    assert sorted(w) == sorted(t) and all(list(w[n].shape) == t[n] for n in t)
    assert "Papunex" in models.architectures()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff,shared", [(20, 30), (20, 9), (20, 20), (8, 40)])
def test_the_shared_experts_pieces_add_up_to_the_whole(monkeypatch, ff, shared, dtype):
    """the loader cuts the shared expert into pieces of the experts' hidden width, zero-padded: the same function"""
    monkeypatch.setattr(Uploader, "_mat_from", lambda self, a32, bits: a32 if a32 is not None else bits)
    monkeypatch.setattr(Uploader, "mat32", lambda self, n: None)
    monkeypatch.setattr(Uploader, "vec", lambda self, n: None)
    conf = papunex.parse_config(config([mamba(mlp=moe(experts=3, top=1, ff=ff, shared=shared))], width=12))
    w = papunex.random_weights(conf, 1)

    class Lc:
        pass
    up, lc = Uploader(None, w, dtype), Lc()
    captured = papunex.PapunexModel._feed_forward(up, lc, conf["layers"][0]["mlp"], "l0.mlp.")
    assert lc.shared == -(-shared // ff)
    U, Dn = captured["up"].reshape(3 + lc.shared, ff, 12), captured["down"].reshape(3 + lc.shared, 12, ff)
    h = np.random.default_rng(2).standard_normal((5, 12))
    got = sum(R.squared_relu_ff(h, U[3 + j], Dn[3 + j]) for j in range(lc.shared))
    assert np.allclose(got, R.squared_relu_ff(h, w["l0.mlp.shared.up"], w["l0.mlp.shared.down"]))
    assert np.array_equal(U[1], w["l0.mlp.e1.up"]) and np.array_equal(Dn[2], w["l0.mlp.e2.down"])
