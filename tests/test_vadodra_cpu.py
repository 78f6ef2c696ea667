"""Pins the plain Vadodra reference (tests/vadodra_ref.py) with cases small enough to do by hand, and checks the package's host-side parts
(configuration, tensor inventory, frequency table, stacked matrices) against it.  No GPU."""
import numpy as np
import pytest

from crabml_b200 import models, rotary, vadodra
from crabml_b200.capi import TensorError
from crabml_b200.seqmodel import Uploader
from tests import vadodra_ref as R
from tests.vadodra_common import config, dense, latent, mixed_config, window


def test_layer_norm_takes_the_mean_off_and_has_eps_inside_the_root():
    x = np.array([[1.0, 3.0, 5.0, 11.0]])
    assert np.allclose(R.layer_norm(x, np.array([1.0, 2.0, 1.0, 1.0]), 2.0), np.array([[-4.0, -4.0, 0.0, 6.0]]) / np.sqrt(14.0 + 2.0))
    assert np.allclose(R.rms_norm(np.array([3.0, 4.0]), np.array([2.0, 1.0]), 2.5), np.array([6.0, 4.0]) / np.sqrt(15.0))


def test_rotations_pair_neighbours_or_halves_and_leave_the_rest():
    rot = {"dims": 4, "base": 100.0}
    x = np.zeros((4, 5)); x[3] = [1.0, 2.0, 3.0, 4.0, 9.0]
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    assert np.allclose(R.rotate_neighbours(x, rot)[3], [np.cos(a0) - 2 * np.sin(a0), 2 * np.cos(a0) + np.sin(a0), 3 * np.cos(a1) - 4 * np.sin(a1), 4 * np.cos(a1) + 3 * np.sin(a1), 9.0])
    assert np.allclose(R.rotate_halves(x, rot)[3], [np.cos(a0) - 3 * np.sin(a0), 2 * np.cos(a1) - 4 * np.sin(a1), 3 * np.cos(a0) + np.sin(a0), 4 * np.cos(a1) + 2 * np.sin(a1), 9.0])
    assert np.allclose(R.rotate_halves(x[3:], rot), x[3:])               # position 0 does not turn
    slow = dict(rot, scaling={"factor": 3.0})
    assert np.allclose(R.rotate_neighbours(x, slow)[3, :2], [np.cos(1.0) - 2 * np.sin(1.0), 2 * np.cos(1.0) + np.sin(1.0)])


@pytest.mark.parametrize("dims,base,factor", [(2, 10.0, None), (6, 100.0, 4.0), (64, 3e6, 2.5), (40, 2e5, 8.0)])
def test_frequency_table_of_the_package_is_the_reference_rule(dims, base, factor):
    rot = {"dims": dims, "base": base}
    if factor:
        rot["scaling"] = {"factor": factor}
    f, mag = rotary.table_of(rot)
    assert mag == 1.0 and f.dtype == np.float32 and np.allclose(f, [R.frequency(i, rot) for i in range(dims // 2)], rtol=1e-7)
    # the other rules are still told apart by their keys
    assert rotary.table_of({"dims": 8, "base": 1e4, "scaling": {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 2.0}})[1] > 1.0


def test_window_counts_the_query_itself():
    k = np.zeros((6, 1, 1)); q = np.zeros((6, 1, 1))
    v = np.arange(6.0).reshape(6, 1, 1) ** 2
    out = R.window_attention(q, k, v, 1.0, 3)[:, 0, 0]
    assert np.allclose(out, [0.0, 0.5, 5.0 / 3, 14.0 / 3, 29.0 / 3, 50.0 / 3])
    assert np.allclose(R.window_attention(q, k, v, 1.0, 1)[:, 0, 0], v[:, 0, 0])


def test_query_heads_share_key_heads_as_neighbours():
    rng = np.random.default_rng(0)
    k, v = rng.standard_normal((1, 2, 3)), rng.standard_normal((1, 2, 2))
    out = R.window_attention(rng.standard_normal((1, 6, 3)), k, v, 1.0, 4)
    assert np.allclose(out[0], v[0, [0, 0, 0, 1, 1, 1]])


def test_values_are_the_keys_before_norm_and_rotation():
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "scale": 1.0, "mask": {"size": 1}, "rot": {"dims": 2, "base": 10.0}}
    w = {"m.q": np.ones((2, 2)), "m.k": np.eye(2), "m.q.norm": np.ones(2), "m.k.norm": np.array([7.0, 5.0]), "m.o": np.eye(2)}
    h = np.array([[3.0, 4.0], [1.0, -2.0], [0.5, 0.25]])
    assert np.allclose(R.attention(h, w, "m.", m, 1e-6), h)              # each position sees itself alone and returns its own raw key


def test_query_and_key_norm_weights_enter_the_scores():
    m = {"heads": 2, "kv_heads": 1, "dim": 2, "scale": 0.5, "mask": {"size": 9}, "rot": {"dims": 2, "base": 10.0}}
    rng = np.random.default_rng(1)
    w = {"m.q": rng.standard_normal((4, 3)), "m.k": rng.standard_normal((2, 3)), "m.q.norm": np.array([1.5, 0.5]), "m.k.norm": np.array([2.0, 3.0]), "m.o": np.eye(4)}
    h = rng.standard_normal((3, 3))
    out = R.attention(h, w, "m.", m, 0.1)

    def unit(v, g):
        return v / np.sqrt((v * v).mean() + 0.1) * g

    def turn(v, a):
        return np.array([v[0] * np.cos(a) - v[1] * np.sin(a), v[1] * np.cos(a) + v[0] * np.sin(a)])
    raw = h @ w["m.k"].T
    ks = [turn(unit(raw[j], w["m.k.norm"]), j) for j in range(3)]
    for hh in range(2):
        q = turn(unit(w["m.q"][2 * hh:2 * hh + 2] @ h[2], w["m.q.norm"]), 2)
        e = np.exp([0.5 * (q @ kk) for kk in ks])
        assert np.allclose(out[2, 2 * hh:2 * hh + 2], (e / e.sum()) @ raw)


def _identity_latent():
    """one head; queries and output pass the input's first columns on"""
    D = 4
    m = {"heads": 1, "dim": 2, "rot_dim": 2, "vdim": 2, "kv_rank": 2, "scale": 1.0, "rot": {"dims": 2, "base": 10.0}}
    w = {"m.q": np.zeros((4, D)), "m.dkv": np.eye(4, D), "m.dkv.norm": np.ones(2), "m.uk": np.eye(2), "m.uv": np.eye(2), "m.g": np.zeros((1, D)), "m.o": np.eye(D, 2)}
    return m, w


def test_latent_attention_is_causal_and_gated_by_one_number_per_head():
    m, w = _identity_latent()
    h = np.array([[1.0, 0.0, 0, 0], [0.0, 1.0, 0, 0], [1.0, 1.0, 0, 0]])
    rows = R.latent_rows(h, w, "m.", m, 1e-9)
    out = R.latent_attention(h, rows, w, "m.", m)                        # all scores 0: the mean of the values so far, gated by 1/2
    for i in range(3):
        assert np.allclose(out[i, :2], rows[0][:i + 1].mean(0) / 2)
    w["m.g"] = np.array([[3.0, -1.0, 0, 0]])
    assert np.allclose(R.latent_attention(h, rows, w, "m.", m)[:, :2], out[:, :2] * 2 * R.sigmoid(h @ w["m.g"].T))


def test_the_rotated_key_part_is_not_normed_and_the_latent_is():
    m, w = _identity_latent()
    c, r = R.latent_rows(np.array([[3.0, 4.0, 5.0, 6.0]]), w, "m.", m, 0.0)
    assert np.allclose(c, np.array([[3.0, 4.0]]) / np.sqrt(12.5)) and np.allclose(r, [[5.0, 6.0]])


def test_latent_score_scale_covers_both_parts():
    m, w = _identity_latent()
    m["scale"] = 0.5
    w["m.q"] = np.eye(4)
    h = np.array([[1.0, 0.0, 2.0, 0.0], [1.0, 0.0, 3.0, 0.0]])
    c, r = R.latent_rows(h, w, "m.", m, 0.0)
    qr = [3.0 * np.cos(1.0), 3.0 * np.sin(1.0)]
    e = np.exp([(h[1, :2] @ c[j] + qr @ r[j]) * 0.5 for j in range(2)])
    assert np.allclose(R.latent_attention(h, (c, r), w, "m.", m)[1, :2], (e / e.sum() @ c) * 0.5)


def test_the_gated_unit_clamps_the_gate_from_above_only_and_the_other_from_both_sides():
    def unit(g, u):
        return float(R.clamped_unit(np.array(g), np.array(u), 2.0))
    s = R.sigmoid
    assert np.isclose(unit(1.0, 0.5), s(1.702) * 1.5)
    assert np.isclose(unit(9.0, 0.5), 2 * s(3.404) * 1.5) and np.isclose(unit(-9.0, 0.5), -9 * s(-9 * 1.702) * 1.5)
    assert np.isclose(unit(1.0, 9.0), s(1.702) * 3.0) and np.isclose(unit(1.0, -9.0), s(1.702) * -1.0)


def test_sublayers_read_one_norm_and_the_head_is_the_unscaled_table():
    conf = config([window(mlp=dense(9))])
    w = vadodra.random_weights(vadodra.parse_config(conf), 5)
    taps = []
    logits = R.forward(conf, w, [4, 8, 15], taps)
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    x = w["embed"][[4, 8, 15]] * 5.0
    h = R.layer_norm(x, w["l0.norm1"], 1e-5)
    x = x + R.attention(h, w, "l0.mix.", conf["layers"][0]["mixer"], 1e-5) + R.feed_forward(h, w, "l0.mlp.", conf["layers"][0]["mlp"])
    assert np.allclose(taps[0], x) and np.allclose(logits, R.layer_norm(x, w["final.norm"], 1e-5) @ w["embed"].T)


def test_forward_is_causal_and_taps_every_layer():
    conf = mixed_config()
    w = vadodra.random_weights(vadodra.parse_config(conf), 3)
    a = [5, 9, 2, 44, 1, 0, 17, 30, 30, 8, 3, 21, 40]
    b = a[:7] + [31] + a[8:]
    la, lb = R.forward(conf, w, a), R.forward(conf, w, b)
    assert np.allclose(la[:7], lb[:7]) and np.abs(la[7:] - lb[7:]).max() > 1e-3
    taps = []
    R.forward(conf, w, a, taps)
    assert len(taps) == 7 and taps[0].shape == (len(a), conf["width"])


def test_a_shared_cache_is_the_other_layers():
    # the first layer adds nothing (its W_o is zero) and both norms have equal weights: the second layer, reading the first one's cache, is a lone
    # layer with the first one's latent projection
    conf = vadodra.parse_config(config([latent(mlp=None), latent(heads=2, dim=4, vdim=5, scale=0.7, kv_from=0, mlp=None)]))
    w = vadodra.random_weights(conf, 4)
    w["l0.mix.o"] = np.zeros_like(w["l0.mix.o"])
    w["l1.norm1"] = w["l0.norm1"]
    lone = vadodra.parse_config(config([latent(heads=2, dim=4, vdim=5, scale=0.7, mlp=None)]))
    w1 = {n: w[n.replace("l0.", "l0." if "dkv" in n else "l1.")] for n in vadodra.expected_tensors(lone)}
    toks = [3, 9, 1, 50, 9, 9, 20]
    assert np.allclose(R.forward(conf, w, toks), R.forward(lone, w1, toks))


def test_config_defaults_and_refusals():
    c = vadodra.parse_config(mixed_config())
    assert vadodra.parse_config(c) == c                  # parsing what was parsed changes nothing
    assert c["layers"][3]["mlp"] is None and c["layers"][0]["mixer"]["kv_from"] is None and c["layers"][4]["mixer"]["kv_from"] == 0
    assert c["layers"][1]["mixer"]["rot"]["scaling"] == {"factor": 3.0} and "scaling" not in c["layers"][3]["mixer"]["rot"]
    bare = config([window(), latent()])
    del bare["embedding"], bare["layers"][0]["mixer"]["vdim"], bare["layers"][0]["mlp"], bare["layers"][1]["mixer"]["rot"]["dims"]
    p = vadodra.parse_config(bare)
    assert p["embedding"]["scale"] == 1.0 and p["layers"][0]["mixer"]["vdim"] == 10 and p["layers"][0]["mlp"] is None and p["layers"][1]["mixer"]["rot"]["dims"] == 6

    def wrong(layer, **kw):
        layer["mixer"].update(kw)
        return config([layer])
    for bad in (config([latent(kv_from=0)]), config([latent(), latent(kv_from=1)]), config([window(), latent(kv_from=0)]), config([latent(), latent(kv_from=0), latent(kv_from=1)]),
                config([latent(), latent(kv_from=0, kv_rank=15)]), config([latent(), latent(kv_from=0, rot_dim=4)]), config([latent(), latent(kv_from=0, base=499.0)]),
                config([window(kv_heads=4)]), config([window(rot=12)]), config([window(rot=3)]), wrong(window(), vdim=9), wrong(latent(), rot={"dims": 8, "base": 5.0}),
                config([dict(window(), type="mamba2")]), config([window(mlp={"kind": "moe", "ff": 4, "limit": 1.0})]), config([window(mlp=dense(4, 0.0))]),
                dict(mixed_config(), architecture="Other")):
        with pytest.raises(TensorError):
            vadodra.parse_config(bad)


def test_tensor_inventory_and_registry():
    c = vadodra.parse_config(mixed_config())
    t = vadodra.expected_tensors(c)
    assert "head" not in t and t["embed"] == [53, 36] and t["l1.mix.q"] == [60, 36] and t["l1.mix.k"] == [30, 36] and "l1.mix.v" not in t and t["l1.mix.k.norm"] == [10]
    assert t["l0.mix.q"] == [3 * 14, 36] and t["l0.mix.dkv"] == [20, 36] and t["l0.mix.dkv.norm"] == [14] and t["l0.mix.g"] == [3, 36] and t["l0.mix.o"] == [36, 33]
    assert "l4.mix.dkv" not in t and "l4.mix.dkv.norm" not in t and t["l4.mix.uk"] == [20, 14] and t["l4.mix.uv"] == [15, 14] and "l3.mlp.up" not in t and t["l4.mlp.down"] == [36, 17]
    w = vadodra.random_weights(c, 0)
    assert sorted(w) == sorted(t) and all(list(w[n].shape) == t[n] for n in t)
    assert "Vadodra" in models.architectures()


def test_matrices_are_stacked_under_each_other_and_side_by_side(monkeypatch):
    monkeypatch.setattr(Uploader, "_mat_from", lambda self, a32, bits: a32 if a32 is not None else bits)
    a, b = np.arange(6.0).reshape(2, 3), np.arange(4.0).reshape(2, 2)
    up = Uploader(None, {"a": a, "b": b, "c": a + 1}, "float32")
    assert np.array_equal(up.stack(["a", "c"]), np.concatenate([a, a + 1])) and np.array_equal(up.stack(["a", "b"], axis=1), np.concatenate([a, b], 1))
