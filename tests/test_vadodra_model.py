"""The Vadodra runner (config -> weights -> slots -> steps) against the plain reference on small random models: whole prompts,
token-by-token decoding, portions of several sizes, interleaved requests, reused slots, shared caches, window edges, other sizes, greedy
generation and the trace replay tool."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from crabml_b200 import models, vadodra
from crabml_b200.safetensors import write_safetensors
from tests import vadodra_ref as R
from tests.gpu_common import make_device
from tests.vadodra_common import config, dense, latent, mixed_config, rel_err, run_portions, window

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 1e-4, "bfloat16": 6e-2}


@pytest.fixture(scope="module")
def dev():
    d = make_device()
    yield d
    d.close()


def build(dev, conf, seed, dtype="float32", chunk=0, max_seq=0, weights=None):
    c = vadodra.parse_config(conf)
    w = weights or vadodra.random_weights(c, seed)
    return c, w, vadodra.VadodraModel(dev, conf, w, dtype, chunk, max_seq)


def cut(total, portions):
    """portions with their last one filled up to `total`"""
    return portions + [total - sum(portions)] if sum(portions) < total else portions


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [8, 16, 0])
def test_whole_prompt_decode_and_portions_agree_with_the_reference(dev, dtype, chunk):
    c, w, m = build(dev, mixed_config(), 11, dtype, chunk=chunk)
    toks = np.random.default_rng(0).integers(0, c["vocab"], 90).tolist()
    want = R.forward(mixed_config(), w, toks)
    for portions in ([90], [1] * 90, [58] + [1] * 32, [2, 3, 35, 2, 17, 1, 1, 29], [2] * 45, [7, 8, 9, 31, 35]):
        err = rel_err(run_portions(m, toks, portions), want)
        assert err.max() < TOL[dtype], (portions, err.max())
    assert m.stats()["live"] == 0 and m.stats()["slots"] == 1
    m.close()


def test_prompt_and_decoding_agree_with_each_other(dev):
    c, w, m = build(dev, mixed_config(), 19)
    toks = np.random.default_rng(9).integers(0, c["vocab"], 300).tolist()
    whole = run_portions(m, toks, [300])
    for portions in ([1] * 300, [256, 44], [100, 3, 2, 2, 193]):
        assert rel_err(run_portions(m, toks, portions), whole).max() < 5e-5, portions
    m.close()


def test_residual_stream_after_every_layer(dev):
    from crabml_b200 import CudaTensorDevice
    d = CudaTensorDevice(debug_named_tensors=True)
    c, w, m = build(d, mixed_config(), 21)
    toks = [3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5]
    taps = []
    R.forward(mixed_config(), w, toks, taps)
    assert len(taps) == len(c["layers"])
    s = m.open(); m.step(s, toks, []); m.close_seq(s)
    for i, want in enumerate(taps):
        got = d.dump_debug_tensor(f"layer:{i}:0").reshape(len(toks), -1)
        assert np.abs(got - want).max() < 5e-5 * max(1.0, np.abs(want).max()), i
    m.close(); d.close()


def test_first_tokens_and_single_token_sequence(dev):
    c, w, m = build(dev, mixed_config(), 12)
    for toks in ([5], [5, 9], [0, 0, 0, 0], [52, 0]):
        want = R.forward(mixed_config(), w, toks)
        assert rel_err(run_portions(m, toks, [len(toks)]), want).max() < TOL["float32"]
        assert rel_err(run_portions(m, toks, [1] * len(toks)), want).max() < TOL["float32"]
    m.close()


def test_interleaved_requests_equal_each_alone_and_slots_are_reused(dev):
    c, w, m = build(dev, mixed_config(), 13, chunk=8)
    rng = np.random.default_rng(1)
    A, B, Cq = (rng.integers(0, c["vocab"], n).tolist() for n in (41, 17, 29))
    alone = {k: run_portions(m, t, [len(t)]) for k, t in (("A", A), ("B", B), ("C", Cq))}
    sa, sb = m.open(), m.open()
    assert (sa, sb) == (0, 1)
    got = {"A": [], "B": [], "C": []}
    got["A"].append(m.step(sa, A[:20], range(20))); got["B"].append(m.step(sb, B[:3], range(3)))
    got["A"].append(m.step(sa, A[20:21], [0])); got["B"].append(m.step(sb, B[3:], range(14)))
    m.close_seq(sb)
    sc = m.open()                                             # takes B's slot: its rings hold B's leftovers
    assert sc == 1
    got["C"].append(m.step(sc, Cq[:2], range(2))); got["A"].append(m.step(sa, A[21:], range(20))); got["C"].append(m.step(sc, Cq[2:], range(27)))
    for k in got:
        assert rel_err(np.concatenate(got[k]), alone[k]).max() < 5e-5, k
    for k, t in (("A", A), ("B", B), ("C", Cq)):
        assert rel_err(np.concatenate(got[k]), R.forward(mixed_config(), w, t)).max() < TOL["float32"]
    m.close_seq(sa); m.close_seq(sc)
    assert m.stats() == {"slots": 2, "live": 0, "state_bytes_per_slot": m.stats()["state_bytes_per_slot"]}
    m.close()


def test_state_of_a_slot_is_what_the_config_says(dev):
    c, w, m = build(dev, mixed_config(), 13, chunk=8, max_seq=100)
    latents = 100 * (14 + 6) + 100 * (9 + 4)                  # two caches of their own; the layers that share one hold nothing
    windows = 2 * ((6 + 8) * 30 + (11 + 8) * 24 + (0 + 8) * 10)
    assert m.stats()["state_bytes_per_slot"] == 4 * (latents + windows)
    m.close()
    # a window that reaches past the longest sequence takes no more rows than that
    c, w, m = build(dev, config([window(size=5000)]), 13, chunk=8, max_seq=100)
    assert m.stats()["state_bytes_per_slot"] == 4 * 2 * 100 * 30
    m.close()


def test_long_decoding(dev):
    conf = config([window(size=33), latent(mlp=None), window(heads=3, kv_heads=1, dim=8, size=70, rot=8), latent(heads=2, kv_from=1)])
    c, w, m = build(dev, conf, 14, chunk=32)
    toks = np.random.default_rng(2).integers(0, c["vocab"], 330).tolist()
    want = R.forward(conf, w, toks)
    assert rel_err(run_portions(m, toks, [30] + [1] * 300), want).max() < TOL["float32"]
    assert rel_err(run_portions(m, toks, [3, 4, 1, 2] * 33), want).max() < TOL["float32"]
    m.close()


def test_the_cache_is_sized_by_the_token_budget(dev):
    for conf in (config([latent(), window(), latent(kv_from=0)]), config([window(size=40)]), config([window(size=9999)])):
        c, w, m = build(dev, conf, 18, chunk=8, max_seq=40)
        toks = np.random.default_rng(5).integers(0, c["vocab"], 41).tolist()
        assert rel_err(run_portions(m, toks[:40], [33, 7]), R.forward(conf, w, toks[:40])).max() < TOL["float32"]
        s = m.open()
        m.step(s, toks[:40], [])
        with pytest.raises(vadodra.TensorError):
            m.step(s, toks[40:], [0])                         # the 41st token does not fit
        m.close_seq(s)
        m.close()
    conf = config([window(size=39)])                          # a window inside the budget: the ring laps, sequences go on for ever
    c, w, m = build(dev, conf, 18, chunk=8, max_seq=40)
    toks = np.random.default_rng(6).integers(0, c["vocab"], 150).tolist()
    want = R.forward(conf, w, toks)
    for portions in ([150], [60] + [1] * 90):
        assert rel_err(run_portions(m, toks, portions), want).max() < TOL["float32"]
    m.close()


# ---- one token that alone decides ------------------------------------------------------------------------------------------------------------
def _recall_model(kind, size=0):
    """One mixer (one head) whose scores are 0 but for the key of token id 1, which every query scores with 60 or more; its value carries a mark
    to the logit of id 2.  Coordinates come in pairs (c, -c), so the layer norm only scales: pair 0 says `ordinary`, pair 1 `id 1`, pair 2 is
    constant, pair 3 holds the mark."""
    if kind == "window":
        layer = window(heads=1, kv_heads=1, dim=4, size=size, rot=2, base=10.0, factor=None, scale=15.0, mlp=None)
    else:
        layer = latent(heads=1, dim=2, rot_dim=2, vdim=2, kv_rank=2, scale=1.0, base=10.0, mlp=None)
    conf = config([layer], width=8, vocab=3, eps=1e-6, embed_scale=1.0)
    w = {n: np.zeros(s, np.float32) for n, s in vadodra.expected_tensors(vadodra.parse_config(conf)).items()}
    w["embed"][:] = [[1, -1, 0, 0, 1, -1, 0, 0], [0, 0, 1, -1, 1, -1, 0, 0], [0, 0, 0, 0, 0, 0, 1, -1]]
    w["l0.norm1"][:] = w["final.norm"][:] = 1
    if kind == "window":
        w["l0.mix.q"][3, 4] = 1
        w["l0.mix.k"][2, 0] = w["l0.mix.k"][3, 2] = 1
        w["l0.mix.q.norm"][:] = w["l0.mix.k.norm"][:] = 1
        w["l0.mix.o"][6, 3], w["l0.mix.o"][7, 3] = 1, -1
    else:
        w["l0.mix.q"][0, 4] = 64.0
        w["l0.mix.dkv"][0, 0] = w["l0.mix.dkv"][1, 2] = 1
        w["l0.mix.dkv.norm"][:] = 1
        w["l0.mix.uk"][0, 1] = 1
        w["l0.mix.uv"][0, 1] = 1
        w["l0.mix.o"][6, 0], w["l0.mix.o"][7, 0] = 2, -2          # the gate is one half
    return conf, w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("j_star", [0, 255, 256, 300])
def test_a_far_token_decides_prompts_and_decoded_tokens(dev, dtype, j_star):
    T = 900
    conf, w = _recall_model("latent")
    c, w, m = build(dev, conf, 0, dtype, weights=w)
    toks = [0] * T
    toks[j_star] = 1
    want = R.forward(conf, w, toks)
    for portions in ([T], [820] + [1] * 80, [257, 255, 2, 386]):
        got = run_portions(m, toks, portions)
        assert rel_err(got, want).max() < (1e-3 if dtype == "float32" else 2e-2), portions
        for i in (j_star, 600, T - 1):
            assert got[i, 2] > 2.5
        if j_star:
            assert abs(got[j_star - 1, 2]) < 1e-3             # nobody before it sees it
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [1, 2, 37, 255, 256, 257])
def test_a_token_leaves_the_window_at_its_edge_in_prompts_and_decoded(dev, dtype, size):
    T = 600
    conf, w = _recall_model("window", size)
    c, w, m = build(dev, conf, 0, dtype, weights=w)
    for j_star in (0, 200, 256):
        toks = [0] * T
        toks[j_star] = 1
        seen = (np.arange(T) >= j_star) & (np.arange(T) < j_star + size)
        for portions in ([T], [max(1, j_star + size - 3)] + [1] * 6, [j_star + 1] + [2] * 20, [257, 255, 2]):
            got = run_portions(m, toks, cut(T, portions))
            assert (got[seen, 2] > 2.5).all() and np.abs(got[~seen, 2]).max() < 1e-3, (j_star, portions)
    m.close()


CONFIGS = {
    "one_of_everything": config([window(heads=1, kv_heads=1, dim=2, size=1, rot=2, mlp=dense(1)), latent(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1, mlp=dense(1))], width=8, vocab=19,
                                embed_scale=1.0),
    "every_layer_shares_the_first": config([latent(mlp=None)] + [latent(heads=h, dim=3 + h, vdim=2 * h, scale=0.2 * h, kv_from=0, mlp=dense(8 * h)) for h in (1, 2, 4)]),
    "windows_only": config([window(size=s, heads=h, kv_heads=g, dim=d, rot=r, factor=f) for s, h, g, d, r, f in ((3, 2, 1, 6, 6, 2.0), (64, 4, 4, 8, 2, None), (65, 12, 2, 4, 4, 0.5), (200, 7, 7, 3, 2, 9.0))]),
    "mixers_only": config([window(mlp=None), latent(mlp=None), window(size=11, mlp=None)], embed_scale=0.25),
    "heads_that_do_not_fill_a_tile": config([window(heads=33, kv_heads=1, dim=4, rot=2), window(heads=21, kv_heads=7, dim=6, rot=2, size=30)], width=40, vocab=33),
    "many_heads": config([latent(heads=70, dim=2, rot_dim=2, vdim=2, kv_rank=5, mlp=None), latent(heads=33, dim=2, rot_dim=2, vdim=3, kv_rank=5, kv_from=0)], width=40, vocab=33),
    "aligned_for_tensor_cores": config([latent(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, mlp=dense(192, 1.1)), window(heads=6, kv_heads=2, dim=32, size=45, rot=16, mlp=dense(320)),
                                        latent(heads=2, dim=64, rot_dim=16, vdim=64, kv_rank=64, kv_from=0, mlp=dense(128)), window(heads=2, kv_heads=1, dim=64, size=100, rot=64, mlp=None)],
                                       width=128, vocab=256),
    "wide_rows": config([latent(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=40), window(heads=10, kv_heads=5, dim=48, size=50, rot=48, mlp=dense(700, 3.0))], width=1064, vocab=64),
}


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes_and_layer_orders(dev, name, dtype):
    c, w, m = build(dev, CONFIGS[name], 20, dtype, chunk=64)
    toks = np.random.default_rng(3).integers(0, c["vocab"], 110).tolist()
    want = R.forward(CONFIGS[name], w, toks)
    for portions in ([110], [40, 7, 2, 1, 60], [64, 46], [95] + [1] * 15):
        err = rel_err(run_portions(m, toks, portions), want)
        assert err.max() < TOL[dtype], (name, portions, err.max())
    m.close()


def random_config(seed):
    """sizes drawn so that odd widths and head sizes, both mixers in every place, shared caches and layers without a feed-forward all come up over
    the seeds"""
    rng = np.random.default_rng(7000 + seed)
    layers, owners = [], []
    for i in range(int(rng.integers(1, 7))):
        mlp = None if rng.random() < 0.25 else dense(int(rng.integers(1, 150)), float(rng.uniform(0.2, 5.0)))
        if rng.random() < 0.5:
            g, d = int(rng.integers(1, 5)), int(rng.integers(2, 40))
            layers.append(window(heads=g * int(rng.integers(1, 6)), kv_heads=g, dim=d, size=int(rng.integers(1, 100)), rot=2 * int(rng.integers(1, d // 2 + 1)),
                                 base=float(rng.choice([20.0, 1e4, 3e6])), factor=float(rng.choice([0.0, 0.5, 6.0])), scale=float(rng.uniform(0.05, 0.5)), mlp=mlp))
            continue
        kw = dict(heads=int(rng.integers(1, 12)), dim=int(rng.integers(2, 40)), vdim=int(rng.integers(1, 40)), scale=float(rng.uniform(0.05, 0.5)), mlp=mlp)
        if owners and rng.random() < 0.5:
            j = int(rng.choice(owners))
            src = layers[j]["mixer"]
            layers.append(latent(kv_rank=src["kv_rank"], rot_dim=src["rot_dim"], base=src["rot"]["base"], kv_from=j, **kw))
        else:
            owners.append(i)
            layers.append(latent(kv_rank=int(rng.integers(3, 60)), rot_dim=2 * int(rng.integers(1, 16)), base=float(rng.choice([50.0, 1e4, 3e6])), **kw))
    return config(layers, width=int(rng.integers(8, 90)), vocab=int(rng.integers(8, 200)), eps=float(rng.choice([1e-6, 1e-5, 1e-3])), embed_scale=float(rng.choice([1.0, 4.0, 11.0])))


@pytest.mark.parametrize("seed", range(30))
def test_random_configurations(dev, seed):
    conf = random_config(seed)
    c, w, m = build(dev, conf, seed, "float32", chunk=int(np.random.default_rng(seed).choice([8, 32, 70])))
    toks = np.random.default_rng(seed).integers(0, c["vocab"], 110).tolist()
    want = R.forward(conf, w, toks)
    for portions in ([110], [75] + [1] * 35, [2, 33, 3, 65, 7]):
        err = rel_err(run_portions(m, toks, portions), want)
        assert err.max() < 3 * TOL["float32"] and np.median(err) < TOL["float32"] / 2, (seed, portions, err.max())
    m.close()
    c, w, m = build(dev, conf, seed, "bfloat16", chunk=32)
    err = rel_err(run_portions(m, toks, [37, 1, 72]), want)
    assert np.median(err) < TOL["bfloat16"] and err.max() < 5 * TOL["bfloat16"], (seed, np.median(err), err.max())
    m.close()


def test_greedy_generation_through_the_runner(dev):
    c, w, m = build(dev, mixed_config(), 15)
    prompt = [3, 1, 4, 1, 5, 9, 2, 6]
    s = m.open()
    ids = m.generate_greedy(s, prompt, 24)
    m.close_seq(s)
    assert len(ids) == 24
    # the same chain through the step interface (what a host-side sampler would do): the LAST maximum, as the device sampler takes
    s = m.open()
    lg = m.step(s, prompt, [len(prompt) - 1])[0]
    chain = []
    for _ in range(24):
        t = int(len(lg) - 1 - np.argmax(lg[::-1]))
        chain.append(t)
        lg = m.step(s, [t], [0])[0]
    m.close_seq(s)
    assert ids == chain
    # and against the reference wherever its own choice is not a close call
    seq = list(prompt)
    for t in ids:
        ref = R.forward(mixed_config(), w, seq)[-1]
        top2 = np.sort(ref)[-2:]
        if top2[1] - top2[0] > 1e-3:
            assert t == int(np.argmax(ref))
        seq.append(t)
    with pytest.raises(vadodra.TensorError):
        m.step(s, [1], [0])                                   # a closed slot is refused
    m.close()


def test_trace_replay_tool(dev, tmp_path):
    c = vadodra.parse_config(mixed_config())
    w = vadodra.random_weights(c, 16)
    mdir = os.path.join(tmp_path, "model"); outd = os.path.join(tmp_path, "out")
    os.makedirs(mdir)
    with open(os.path.join(mdir, "config.json"), "w") as f:
        json.dump(mixed_config(), f)
    write_safetensors(os.path.join(mdir, "model.safetensors"), w)
    assert models.architecture_of(mdir) == "Vadodra"
    rng = np.random.default_rng(4)
    a, b = rng.integers(0, c["vocab"], 25).tolist(), rng.integers(0, c["vocab"], 6).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[20:22], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[22:], "want": [2]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [1, 5]}], "end": ["b"]}]
    for dtype in ("float32", "bfloat16"):
        p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", mdir, "--dtype", dtype, "--out", outd, "--max-tokens", "64"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        assert not os.path.exists(os.path.join(outd, "1.f32"))
        ra, rb = R.forward(mixed_config(), w, a), R.forward(mixed_config(), w, b)
        for step, want in ((0, ra[[0, 19]]), (2, ra[[24]]), (3, rb[[1, 5]])):
            got = np.fromfile(os.path.join(outd, f"{step}.f32"), "<f4").reshape(-1, c["vocab"])
            assert rel_err(got, want).max() < TOL[dtype]


def test_loader_refuses_a_model_that_does_not_fit_its_config(dev):
    c = vadodra.parse_config(mixed_config())
    w = vadodra.random_weights(c, 17)
    for name, change in (("l0.mix.g", None), ("l2.mix.dkv.norm", None), ("l1.mix.k.norm", None), ("l4.mlp.down", lambda a: a[:, :-1]), ("l4.mix.uk", lambda a: a[:, :-1]),
                         ("l3.mix.k", lambda a: a[:-1]), ("l5.norm1", lambda a: a[:-1])):
        bad = dict(w)
        if change is None:
            del bad[name]
        else:
            bad[name] = change(bad[name])
        with pytest.raises(vadodra.TensorError):
            vadodra.VadodraModel(dev, mixed_config(), bad, "float32")
