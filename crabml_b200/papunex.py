"""The Papunex decoder family: configuration, weight loading and the Python handle on its C++ runner
(crabml_b200/csrc/host/papunex_runner.cpp; the stack is described in include/crabml_papunex.h).

A model folder holds config.json and model.safetensors.  config.json gives every size and every constant that can differ between
models of the family: `vocab`, `width`, `embedding.scale`, `norm.eps`, `logit_softcap` and `layers`, a list whose entries name the layer's
mixer (`type`: "latent_attention" or "mamba2"), the mixer's sizes (`mixer`) and its feed-forward (`mlp`: kind "dense" or "moe", or null).
A latent-attention mixer with `kv_from` reads the cache of that earlier layer and has no projection into the latent of its own.  A moe has
`router` (`experts`, `top`, `scale`), `expert.ff` and, optionally, `shared.ff`.  Tensor names: `embed`, `head`, `final.norm`, and per layer i
`l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`, `l<i>.mlp.*`.

Precision: `dtype="bfloat16"` keeps the matrices of the dense products in bfloat16 (activations are rounded to bfloat16 at the input
of a product, sums are 32-bit); `dtype="float32"` widens them and every product is a true 32-bit one.  In both modes the residual
stream, norms, rotations, attention scores and sums (with the key / value up-projections folded into them), gates, routers, step sizes,
decays, the convolution and all recurrent state are 32-bit.
"""
from __future__ import annotations

import ctypes as C
import json
import os

import numpy as np

from . import capi, rotary
from .capi import CudaError, TensorError
from .safetensors import bf16_to_f32, f32_to_bf16, read_safetensors
from .seqmodel import STATE_SPACE_FIELDS, SeqModel, Uploader, handle_of, parse_state_space, state_space_tensors
from .tensor import CudaTensorDevice

ARCHITECTURE = "Papunex"
MIXERS = {"latent_attention": 0, "mamba2": 1}
FF_KINDS = {"dense": 1, "moe": 2}


# ---- configuration ----------------------------------------------------------------------------------------------------------------
def parse_config(conf: dict) -> dict:
    """Validates a config.json dict and fills the optional keys, so that the rest of the code reads one shape of dict."""
    if conf.get("architecture", ARCHITECTURE) != ARCHITECTURE:
        raise TensorError(f"not a {ARCHITECTURE} config: architecture = {conf.get('architecture')!r}")
    out = {"architecture": ARCHITECTURE, "vocab": int(conf["vocab"]), "width": int(conf["width"]),
           "embedding": {"scale": float((conf.get("embedding") or {}).get("scale", 1.0))}, "norm": {"eps": float(conf["norm"]["eps"])},
           "logit_softcap": float(conf.get("logit_softcap") or 0.0), "layers": []}
    for i, L in enumerate(conf["layers"]):
        at = f"layer {i}"
        if L["type"] not in MIXERS:
            raise TensorError(f"{at}: unknown mixer type {L['type']!r}")
        m = _latent_mixer(L["mixer"], i, out["layers"]) if L["type"] == "latent_attention" else parse_state_space(L["mixer"], at)
        out["layers"].append({"type": L["type"], "mixer": m, "mlp": _mlp(L.get("mlp"), at)})
    return out


def _latent_mixer(raw: dict, i: int, before: list) -> dict:
    at = f"layer {i}"
    m = {k: int(raw[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
    m["scale"] = float(raw["scale"])
    r = raw.get("rot")
    m["rot"] = {"dims": int(r.get("dims", m["rot_dim"])), "base": float(r["base"])} if r and m["rot_dim"] > 0 else None
    if m["rot"] and (m["rot"]["dims"] > m["rot_dim"] or m["rot"]["dims"] % 2):
        raise TensorError(f"{at}: rot.dims must be even and at most rot_dim")
    j = raw.get("kv_from")
    m["kv_from"] = None if j is None else int(j)
    if j is not None:
        if not 0 <= m["kv_from"] < i or before[m["kv_from"]]["type"] != "latent_attention" or before[m["kv_from"]]["mixer"]["kv_from"] is not None:
            raise TensorError(f"{at}: kv_from = {j} names no earlier latent-attention layer with a cache of its own")
        src = before[m["kv_from"]]["mixer"]
        if any(src[k] != m[k] for k in ("kv_rank", "rot_dim", "rot")):
            raise TensorError(f"{at}: kv_rank, rot_dim and rotation must equal those of layer {j}")
    return m


def _mlp(mlp, at: str):
    if mlp is None:
        return None
    kind = mlp.get("kind")
    if kind == "dense":
        return {"kind": "dense", "ff": int(mlp["ff"])}
    if kind != "moe":
        raise TensorError(f"{at}: unknown feed-forward kind {kind!r}")
    r = mlp["router"]
    out = {"kind": "moe", "expert": {"ff": int(mlp["expert"]["ff"])},
           "router": {"experts": int(r["experts"]), "top": int(r["top"]), "scale": float(r.get("scale", 1.0))},
           "shared": {"ff": int(mlp["shared"]["ff"])} if mlp.get("shared") else None}
    if not 1 <= out["router"]["top"] <= out["router"]["experts"]:
        raise TensorError(f"{at}: router.top must lie between 1 and router.experts")
    return out


def expected_tensors(conf: dict) -> dict:
    """name -> shape of every tensor a model of this config has"""
    D, V = conf["width"], conf["vocab"]
    t = {"embed": [V, D], "head": [V, D], "final.norm": [D]}
    for i, L in enumerate(conf["layers"]):
        m, mlp, p = L["mixer"], L["mlp"], f"l{i}."
        q = p + "mix."
        t[p + "norm1"] = [D]
        if L["type"] == "latent_attention":
            H, dn, dr, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            t.update({q + "q": [H * (dn + dr), D], q + "uk": [H * dn, kr], q + "uv": [H * dv, kr], q + "sink": [H], q + "g": [H * dv, D], q + "o": [D, H * dv]})
            if m["kv_from"] is None:
                t.update({q + "dkv": [kr + dr, D], q + "dkv.norm": [kr]})
        else:
            t.update(state_space_tensors(m, q, D))
        if not mlp:
            continue
        t[p + "norm2"] = [D]
        f = p + "mlp."
        if mlp["kind"] == "dense":
            t.update({f + "up": [mlp["ff"], D], f + "down": [D, mlp["ff"]]})
            continue
        ff = mlp["expert"]["ff"]
        t[f + "router"] = [mlp["router"]["experts"], D]
        for e in range(mlp["router"]["experts"]):
            t.update({f"{f}e{e}.up": [ff, D], f"{f}e{e}.down": [D, ff]})
        if mlp["shared"]:
            t.update({f + "shared.up": [mlp["shared"]["ff"], D], f + "shared.down": [D, mlp["shared"]["ff"]], f + "shared.sg": [1, D]})
    return t


def random_weights(conf: dict, seed: int = 0, scale: float = 1.0) -> dict:
    """Random weights of a config (float32 arrays whose values are exact in bfloat16), sized so that activations stay O(1)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in expected_tensors(conf).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2", "norm"):
            a = 1.0 + 0.1 * rng.standard_normal(shape)
        elif leaf in ("sink", "D"):
            a = rng.standard_normal(shape)
        elif leaf == "A_log":
            a = rng.uniform(-2.0, 1.0, shape)
        elif leaf == "dt_bias":
            a = rng.uniform(-3.0, 0.0, shape)
        elif leaf in ("b", "conv"):
            a = rng.standard_normal(shape) * 0.5
        elif name == "embed":
            a = rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) * (scale / np.sqrt(shape[-1]))
        out[name] = bf16_to_f32(f32_to_bf16(np.asarray(a, np.float32))).reshape(shape)
    return out


# ---- the model on a device ------------------------------------------------------------------------------------------------------------
class PapunexModel(SeqModel):
    """Weights of one model on one device + its runner (sequences, steps and generation: seqmodel.SeqModel).  `weights`: {name: float32
    ndarray} or the pair read_safetensors returns."""

    def __init__(self, device: CudaTensorDevice, conf: dict, weights, dtype: str = "bfloat16", chunk: int = 0, max_seq: int = 0):
        self.device, self.conf, self.dtype = device, parse_config(conf), dtype
        up = Uploader(device, weights, dtype)
        c = self.conf
        up.check(expected_tensors(c))
        nl = len(c["layers"])
        # the embedding scale is folded into the (32-bit) table: one rounding, as when it is applied to the looked-up row
        self.tensors = {"embed": up.table(up.f32("embed") * np.float32(c["embedding"]["scale"])), "final.norm": up.vec("final.norm"), "head": up.mat("head")}
        lcs = (capi.cpr_layer_config * nl)()
        lws = (capi.cpr_layer_weights * nl)()
        for i, L in enumerate(c["layers"]):
            m, mlp, p = L["mixer"], L["mlp"], f"l{i}."
            q, lc = p + "mix.", lcs[i]
            lc.mixer = MIXERS[L["type"]]
            t = {"norm1": up.vec(p + "norm1")}
            if L["type"] == "latent_attention":
                lc.heads, lc.dim, lc.rot_dim, lc.vdim, lc.kv_rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
                lc.kv_from, lc.scale, lc.rot_mag = -1 if m["kv_from"] is None else m["kv_from"], m["scale"], 1.0
                # one product for everything that multiplies the layer's input (the order include/crabml_papunex.h gives)
                t["h_stack"] = up.stack([q + "q", q + "g"] + ([q + "dkv"] if m["kv_from"] is None else []))
                if m["kv_from"] is None:
                    t["dkv_norm"] = up.vec(q + "dkv.norm")
                t.update(up.latent_projections(q, m["heads"], m["dim"], m["kv_rank"]))
                if m["rot"] and m["rot"]["dims"] > 0:
                    freq, mag = rotary.table_of(m["rot"])
                    t["rot_freq"], lc.rot_mag = up.table(freq), mag
                t["o"] = up.mat(q + "o")
            else:
                for key, field in STATE_SPACE_FIELDS.items():
                    setattr(lc, field, m[key])
                t.update(up.state_space(q))
            if mlp:
                t["norm2"] = up.vec(p + "norm2")
                t.update(self._feed_forward(up, lc, mlp, p + "mlp."))
            for k, v in t.items():
                setattr(lws[i], k, handle_of(v))
                self.tensors[f"{p}{k}"] = v                                  # keep alive
        cc = capi.cpr_config(nl, c["width"], c["vocab"], c["norm"]["eps"], c["logit_softcap"], int(chunk), int(max_seq))
        h = C.c_void_p()
        rc = device.lib.cpr_runner_create(device.handle, C.byref(cc), lcs, lws, self.tensors["embed"].buf.handle, self.tensors["final.norm"].buf.handle,
                                          self.tensors["head"].buf.handle, C.byref(h))
        if rc != capi.CC_OK:
            raise (TensorError if rc == capi.CC_ERR_TENSOR else CudaError)(f"cpr_runner_create failed [{rc}]: {device.lib.csr_last_create_error().decode()}")
        self.handle = h
        self.vocab = c["vocab"]
        self._keep = (lcs, lws)

    @staticmethod
    def _feed_forward(up: Uploader, lc, mlp: dict, f: str) -> dict:
        lc.ff_kind = FF_KINDS[mlp["kind"]]
        if mlp["kind"] == "dense":
            lc.ff = mlp["ff"]
            return {"up": up.mat(f + "up"), "down": up.mat(f + "down")}
        r, ff = mlp["router"], mlp["expert"]["ff"]
        lc.ff, lc.experts, lc.top, lc.route_scale = ff, r["experts"], r["top"], r["scale"]
        ups, downs = [f"{f}e{e}.up" for e in range(r["experts"])], [f"{f}e{e}.down" for e in range(r["experts"])]
        t = {"router": up.mat32(f + "router")}
        if mlp["shared"]:
            # the shared expert in pieces of the experts' hidden width, the last one padded with units that add nothing
            lc.shared = -(-mlp["shared"]["ff"] // ff)
            for j in range(lc.shared):
                n = min(ff, mlp["shared"]["ff"] - j * ff)
                ups.append((f + "shared.up", lambda a, j=j, n=n: np.pad(a[j * ff:j * ff + n], ((0, ff - n), (0, 0)))))
                downs.append((f + "shared.down", lambda a, j=j, n=n: np.pad(a[:, j * ff:j * ff + n], ((0, 0), (0, ff - n)))))
            t["shared_gate"] = up.vec(f + "shared.sg")
        return {**t, "up": up.stack(ups), "down": up.stack(downs)}


def load(path: str, device: CudaTensorDevice, dtype: str = "bfloat16", chunk: int = 0, max_seq: int = 0) -> PapunexModel:
    """path: a folder with config.json and model.safetensors"""
    with open(os.path.join(path, "config.json")) as f:
        conf = json.load(f)
    return PapunexModel(device, conf, read_safetensors(os.path.join(path, "model.safetensors")), dtype, chunk, max_seq)
