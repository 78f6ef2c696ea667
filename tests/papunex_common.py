"""Small Papunex configurations for the tests.  Sizes differ from layer to layer and avoid values that would make two of them equal by
accident (head counts, head sizes, value sizes, latent sizes, groups, taps, hidden widths)."""
from tests.meresun_common import rel_err, run_portions  # noqa: F401  (helpers that only drive the runner)


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=20, scale=1.7, shared=30):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def latent(heads=3, dim=8, rot_dim=6, vdim=10, kv_rank=14, scale=0.3, base=500.0, kv_from=None, mlp="default"):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"dims": rot_dim, "base": base}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": dense() if mlp == "default" else mlp}


def mamba(heads=4, vdim=6, state=10, groups=2, conv=3, norm_groups=3, mlp="default"):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups},
            "mlp": moe() if mlp == "default" else mlp}


def config(layers, width=36, vocab=53, eps=1e-5, embed_scale=3.0, softcap=8.0):
    c = {"architecture": "Papunex", "vocab": vocab, "width": width, "embedding": {"scale": embed_scale}, "norm": {"eps": eps}, "layers": layers}
    if softcap:
        c["logit_softcap"] = softcap
    return c


def mixed_config():
    """both mixers, every feed-forward, two caches of their own and two layers that read them with other head counts and sizes; sharing layers
    stand behind other mixers and out of order"""
    return config([mamba(mlp=None), latent(), latent(heads=2, dim=12, rot_dim=4, vdim=7, kv_rank=9, base=60.0, mlp=moe(experts=5, top=3, ff=16, scale=0.6, shared=0)),
                   mamba(heads=6, vdim=5, state=7, groups=3, conv=5, norm_groups=2, mlp=dense(24)), latent(heads=5, dim=4, vdim=3, scale=0.5, kv_from=1, mlp=moe(shared=9)),
                   latent(heads=1, dim=10, rot_dim=4, vdim=16, kv_rank=9, base=60.0, scale=0.2, kv_from=2, mlp=None)])
