"""Shared pieces of the Bezizen tests: small configurations in the parsed-JSON form a checkpoint carries, and the engine builder for the
two backends of seqlm_common (kernel sources under the CPU emulator; the native library on a GPU)."""
import copy

from seqlm_common import BACKENDS, TOL, backend, emu_lib, rel_err  # noqa: F401  (fixtures)


def moe(experts=6, top=3, groups=(3, 2), ff=5, shared=7, scale=1.6):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        d["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def wkv_layer(heads=2, dim=6, rank=5, mlp=None):
    """rank: read by the weight maker only, a checkpoint gives it by its tensors' shapes"""
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "rank": rank}, "mlp": mlp}


def parallel_layer(heads=4, kv_heads=2, dim=8, conv=3, window=5, scale=0.5, coef=0.4, every=3, left=1.2, right=0.7, gheads=3, gdim=6, gvdim=5,
                   tau=4.0, rank=3, mlp=None):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "mask": {"size": window}, "scale": scale,
                 "q_temp": {"coef": coef, "every": every}},
        "right": {"heads": gheads, "dim": gdim, "vdim": gvdim, "tau": tau, "rank": rank}, "left_scale": left, "right_scale": right}, "mlp": mlp}


def model(layers, width=12, vocab=41, eps=1e-5, embed=1.5, streams=2, positions=300, logit_scale=0.6):
    return {"architecture": "Bezizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed}, "streams": streams,
            "max_positions": positions, "logit_scale": logit_scale, "layers": copy.deepcopy(layers)}


def mixed_model(**kw):
    """both mixers, layers with and without feed-forward, three streams"""
    kw.setdefault("streams", 3)
    return model([wkv_layer(mlp=moe()), parallel_layer(mlp=moe(experts=4, groups=None, shared=0, scale=0.8)), wkv_layer(heads=1, dim=9)], **kw)


def make_engine(cfg: dict, weights: dict, backend, dtype="float32", **kw):
    from leopard_b200 import bezizen
    device, lib = backend
    kw.setdefault("page_size", 4)
    kw.setdefault("max_tokens", 32)
    kw.setdefault("max_seqs", 2)
    return bezizen.from_state_dict(cfg, weights, dtype=dtype, device=device, lib=lib, **kw)
