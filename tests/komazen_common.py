"""Shared pieces of the Komazen tests: small configurations in the parsed-JSON form a checkpoint carries, and the engine builder for
the two backends of seqlm_common (kernel sources under the CPU emulator; the native library on a GPU)."""
import copy

from seqlm_common import BACKENDS, TOL, backend, emu_lib, rel_err  # noqa: F401  (fixtures)


def dense(ff=10):
    return {"kind": "dense", "ff": ff}


def latent_layer(heads=2, dim=6, rot_dim=4, vdim=5, q_rank=7, kv_rank=9, window=5, scale=0.4, base=100.0, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}, "mask": {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def attention_layer(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.5, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}, "mlp": mlp}


def model(layers, width=12, vocab=41, eps=1e-5, alpha=1.8, embed=1.5, taps=3):
    return {"architecture": "Komazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "postln_alpha": alpha, "canon": {"taps": taps}, "layers": copy.deepcopy(layers)}


def mixed_model(**kw):
    """both mixers, a latent layer on the first one's latents with other heads and a longer window, layers with and without
    feed-forward"""
    return model([latent_layer(mlp=dense()), attention_layer(), latent_layer(heads=3, dim=4, vdim=3, window=7, scale=0.7, kv_from=0,
                                                                            mlp=dense(ff=7))], **kw)


def make_engine(cfg: dict, weights: dict, backend, dtype="float32", **kw):
    from leopard_b200 import komazen
    device, lib = backend
    kw.setdefault("page_size", 4)
    kw.setdefault("max_tokens", 32)
    kw.setdefault("max_seqs", 2)
    return komazen.from_state_dict(cfg, weights, dtype=dtype, device=device, lib=lib, **kw)
