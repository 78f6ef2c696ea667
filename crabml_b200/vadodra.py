"""The Vadodra decoder family: configuration, weight loading and the Python handle on its C++ runner
(crabml_b200/csrc/host/vadodra_runner.cpp; the stack is described in include/crabml_vadodra.h).

A model folder holds config.json and model.safetensors.  config.json gives every size and every constant that can differ between
models of the family: `vocab`, `width`, `embedding.scale`, `norm.eps` and `layers`, a list whose entries name the layer's mixer (`type`:
"attention" or "latent_attention"), the mixer's sizes (`mixer`) and its feed-forward (`mlp`: kind "dense" with `ff` and `limit`, or null).
An attention mixer has `mask.size`, the window, and its values are its keys as projected, so `vdim` equals `dim`.  A latent-attention mixer
with `kv_from` reads the cache of that earlier layer and has no projection into the latent of its own.  `rot.scaling`, where given, divides the
frequencies (rotary.table_of).  Tensor names: `embed` (which is also the head), `final.norm`, and per layer i `l<i>.norm1`, `l<i>.mix.*`,
`l<i>.mlp.*`.

Precision: `dtype="bfloat16"` keeps the matrices of the dense products in bfloat16 (activations are rounded to bfloat16 at the input
of a product, sums are 32-bit); `dtype="float32"` widens them and every product is a true 32-bit one.  In both modes the residual
stream, norms, rotations, attention scores and sums (with the key / value up-projections folded into them), gates and gated units are
32-bit.
"""
from __future__ import annotations

import ctypes as C
import json
import os

import numpy as np

from . import capi, rotary
from .capi import CudaError, TensorError
from .safetensors import bf16_to_f32, f32_to_bf16, read_safetensors
from .seqmodel import SeqModel, Uploader, handle_of
from .tensor import CudaTensorDevice

ARCHITECTURE = "Vadodra"
MIXERS = {"attention": 0, "latent_attention": 1}
# the gated unit min(g, limit) * sigmoid(alpha min(g, limit)) * (clamp(u) + shift)
UNIT_ALPHA, UNIT_SHIFT = 1.702, 1.0


# ---- configuration ----------------------------------------------------------------------------------------------------------------
def _rot(r, most: int, at: str):
    if not r or int(r.get("dims", 0)) <= 0:
        return None
    out = {"dims": int(r["dims"]), "base": float(r["base"])}
    if r.get("scaling"):
        out["scaling"] = {k: float(v) for k, v in r["scaling"].items() if isinstance(v, (int, float))}
    if out["dims"] > most or out["dims"] % 2:
        raise TensorError(f"{at}: rot.dims must be even and at most {most}")
    return out


def parse_config(conf: dict) -> dict:
    """Validates a config.json dict and fills the optional keys, so that the rest of the code reads one shape of dict."""
    if conf.get("architecture", ARCHITECTURE) != ARCHITECTURE:
        raise TensorError(f"not a {ARCHITECTURE} config: architecture = {conf.get('architecture')!r}")
    out = {"architecture": ARCHITECTURE, "vocab": int(conf["vocab"]), "width": int(conf["width"]),
           "embedding": {"scale": float((conf.get("embedding") or {}).get("scale", 1.0))}, "norm": {"eps": float(conf["norm"]["eps"])}, "layers": []}
    for i, L in enumerate(conf["layers"]):
        if L["type"] not in MIXERS:
            raise TensorError(f"layer {i}: unknown mixer type {L['type']!r}")
        m = _window_mixer(L["mixer"], i) if L["type"] == "attention" else _latent_mixer(L["mixer"], i, out["layers"])
        out["layers"].append({"type": L["type"], "mixer": m, "mlp": _mlp(L.get("mlp"), i)})
    return out


def _window_mixer(raw: dict, i: int) -> dict:
    m = {k: int(raw[k]) for k in ("heads", "kv_heads", "dim")}
    m["vdim"], m["scale"] = int(raw.get("vdim", m["dim"])), float(raw["scale"])
    m["mask"] = {"size": int((raw.get("mask") or {}).get("size", 0))}
    m["rot"] = _rot(raw.get("rot"), m["dim"], f"layer {i}")
    if m["kv_heads"] < 1 or m["heads"] % m["kv_heads"]:
        raise TensorError(f"layer {i}: kv_heads does not divide heads")
    if m["vdim"] != m["dim"]:
        raise TensorError(f"layer {i}: the values are the keys, so vdim must equal dim")
    return m


def _latent_mixer(raw: dict, i: int, before: list) -> dict:
    m = {k: int(raw[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
    m["scale"] = float(raw["scale"])
    m["rot"] = _rot(dict(raw["rot"], dims=raw["rot"].get("dims", m["rot_dim"])), m["rot_dim"], f"layer {i}") if raw.get("rot") and m["rot_dim"] > 0 else None
    j = raw.get("kv_from")
    m["kv_from"] = None if j is None else int(j)
    if j is not None:
        if not 0 <= m["kv_from"] < i or before[m["kv_from"]]["type"] != "latent_attention" or before[m["kv_from"]]["mixer"]["kv_from"] is not None:
            raise TensorError(f"layer {i}: kv_from = {j} names no earlier latent-attention layer with a cache of its own")
        src = before[m["kv_from"]]["mixer"]
        if any(src[k] != m[k] for k in ("kv_rank", "rot_dim", "rot")):
            raise TensorError(f"layer {i}: kv_rank, rot_dim and rotation must equal those of layer {j}")
    return m


def _mlp(mlp, i: int):
    if mlp is None:
        return None
    if mlp.get("kind") != "dense":
        raise TensorError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
    out = {"kind": "dense", "ff": int(mlp["ff"]), "limit": float(mlp["limit"])}
    if out["ff"] < 1 or not out["limit"] > 0.0:
        raise TensorError(f"layer {i}: a feed-forward needs a width and a positive limit")
    return out


def expected_tensors(conf: dict) -> dict:
    """name -> shape of every tensor a model of this (parsed) config has"""
    D, V = conf["width"], conf["vocab"]
    t = {"embed": [V, D], "final.norm": [D]}
    for i, L in enumerate(conf["layers"]):
        m, p = L["mixer"], f"l{i}."
        q = p + "mix."
        t[p + "norm1"] = [D]
        if L["type"] == "attention":
            d = m["dim"]
            t.update({q + "q": [m["heads"] * d, D], q + "k": [m["kv_heads"] * d, D], q + "q.norm": [d], q + "k.norm": [d], q + "o": [D, m["heads"] * d]})
        else:
            H, dn, dr, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            t.update({q + "q": [H * (dn + dr), D], q + "uk": [H * dn, kr], q + "uv": [H * dv, kr], q + "g": [H, D], q + "o": [D, H * dv]})
            if m["kv_from"] is None:
                t.update({q + "dkv": [kr + dr, D], q + "dkv.norm": [kr]})
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            t.update({p + "mlp.gate": [ff, D], p + "mlp.up": [ff, D], p + "mlp.down": [D, ff]})
    return t


def random_weights(conf: dict, seed: int = 0, scale: float = 1.0) -> dict:
    """Random weights of a (parsed) config (float32 arrays whose values are exact in bfloat16), sized so that activations stay O(1)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in expected_tensors(conf).items():
        if name.endswith(("norm1", ".norm")):
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name == "embed":                                        # also the head: rows of unit length
            a = rng.standard_normal(shape) / np.sqrt(shape[-1])
        else:
            a = rng.standard_normal(shape) * (scale / np.sqrt(shape[-1]))
        out[name] = bf16_to_f32(f32_to_bf16(np.asarray(a, np.float32))).reshape(shape)
    return out


# ---- the model on a device ------------------------------------------------------------------------------------------------------------
class VadodraModel(SeqModel):
    """Weights of one model on one device + its runner (sequences, steps and generation: seqmodel.SeqModel).  `weights`: {name: float32
    ndarray} or the pair read_safetensors returns."""

    def __init__(self, device: CudaTensorDevice, conf: dict, weights, dtype: str = "bfloat16", chunk: int = 0, max_seq: int = 0):
        self.device, self.conf, self.dtype = device, parse_config(conf), dtype
        up = Uploader(device, weights, dtype)
        c = self.conf
        up.check(expected_tensors(c))
        nl = len(c["layers"])
        # the embedding scale is folded into the (32-bit) table: one rounding, as when it is applied to the looked-up row; the head is the table without it
        self.tensors = {"embed": up.table(up.f32("embed") * np.float32(c["embedding"]["scale"])), "final.norm": up.vec("final.norm"), "head": up.mat("embed")}
        lcs = (capi.cvd_layer_config * nl)()
        lws = (capi.cvd_layer_weights * nl)()
        for i, L in enumerate(c["layers"]):
            m, mlp, p = L["mixer"], L["mlp"], f"l{i}."
            q, lc = p + "mix.", lcs[i]
            lc.mixer, lc.heads, lc.dim, lc.vdim, lc.scale, lc.rot_mag, lc.kv_from = MIXERS[L["type"]], m["heads"], m["dim"], m["vdim"], m["scale"], 1.0, -1
            t = {"norm": up.vec(p + "norm1")}
            # one product for everything that multiplies the layer's normed input (the order include/crabml_vadodra.h gives)
            if L["type"] == "attention":
                lc.kv_heads, lc.window = m["kv_heads"], m["mask"]["size"]
                stack = [q + "q", q + "k"]
                t.update({"q_norm": up.vec(q + "q.norm"), "k_norm": up.vec(q + "k.norm")})
            else:
                lc.rot_dim, lc.kv_rank = m["rot_dim"], m["kv_rank"]
                stack = [q + "q", q + "g"]
                if m["kv_from"] is None:
                    stack.append(q + "dkv")
                    t["dkv_norm"] = up.vec(q + "dkv.norm")
                else:
                    lc.kv_from = m["kv_from"]
                t.update(up.latent_projections(q, m["heads"], m["dim"], m["kv_rank"]))
            if m["rot"]:
                freq, mag = rotary.table_of(m["rot"])
                t["rot_freq"], lc.rot_mag = up.table(freq), mag
            outs = [q + "o"]
            if mlp:
                lc.ff, lc.glu = mlp["ff"], capi.cc_glu_params(capi.ACT_SWISH, UNIT_ALPHA, mlp["limit"], UNIT_SHIFT)
                stack += [p + "mlp.gate", p + "mlp.up"]
                outs.append(p + "mlp.down")
            t["h_stack"], t["o_stack"] = up.stack(stack), up.stack(outs, axis=1)
            for k, v in t.items():
                setattr(lws[i], k, handle_of(v))
                self.tensors[f"{p}{k}"] = v                                  # keep alive
        cc = capi.cvd_config(nl, c["width"], c["vocab"], c["norm"]["eps"], int(chunk), int(max_seq))
        h = C.c_void_p()
        rc = device.lib.cvd_runner_create(device.handle, C.byref(cc), lcs, lws, self.tensors["embed"].buf.handle, self.tensors["final.norm"].buf.handle,
                                          self.tensors["head"].buf.handle, C.byref(h))
        if rc != capi.CC_OK:
            raise (TensorError if rc == capi.CC_ERR_TENSOR else CudaError)(f"cvd_runner_create failed [{rc}]: {device.lib.csr_last_create_error().decode()}")
        self.handle = h
        self.vocab = c["vocab"]
        self._keep = (lcs, lws)


def load(path: str, device: CudaTensorDevice, dtype: str = "bfloat16", chunk: int = 0, max_seq: int = 0) -> VadodraModel:
    """path: a folder with config.json and model.safetensors"""
    with open(os.path.join(path, "config.json")) as f:
        conf = json.load(f)
    return VadodraModel(device, conf, read_safetensors(os.path.join(path, "model.safetensors")), dtype, chunk, max_seq)
