"""Small Vadodra configurations for the tests.  Sizes differ from layer to layer and avoid values that would make two of them equal by
accident (head counts, head sizes, rotated columns, value sizes, latent sizes, windows, hidden widths, limits)."""
from tests.meresun_common import rel_err, run_portions  # noqa: F401  (helpers that only drive the runner)


def dense(ff=40, limit=0.8):
    return {"kind": "dense", "ff": ff, "limit": limit}


def window(heads=6, kv_heads=3, dim=10, size=7, rot=4, base=200.0, factor=3.0, scale=0.35, mlp="default"):
    r = {"dims": rot, "base": base}
    if factor:
        r["scaling"] = {"factor": factor}
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "mask": {"size": size}, "rot": r},
            "mlp": dense() if mlp == "default" else mlp}


def latent(heads=3, dim=8, rot_dim=6, vdim=11, kv_rank=14, scale=0.3, base=500.0, kv_from=None, mlp="default"):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"dims": rot_dim, "base": base}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": dense() if mlp == "default" else mlp}


def config(layers, width=36, vocab=53, eps=1e-5, embed_scale=5.0):
    return {"architecture": "Vadodra", "vocab": vocab, "width": width, "embedding": {"scale": embed_scale}, "norm": {"eps": eps}, "layers": layers}


def mixed_config():
    """both mixers with and without a feed-forward, three windows, two caches of their own and two layers that read them with other head counts
    and sizes; sharing layers stand behind other mixers and out of order"""
    return config([latent(), window(), latent(heads=2, dim=12, rot_dim=4, vdim=7, kv_rank=9, base=60.0, mlp=dense(25, 2.5)), window(heads=4, kv_heads=4, dim=6, size=12, rot=6, base=90.0,
                  factor=None, mlp=None), latent(heads=5, dim=4, vdim=3, scale=0.5, kv_from=0, mlp=dense(17, 0.4)), window(heads=8, kv_heads=2, dim=5, size=1, rot=2, mlp=dense(12)),
                  latent(heads=1, dim=10, rot_dim=4, vdim=16, kv_rank=9, base=60.0, scale=0.2, kv_from=2, mlp=None)])
