"""Komazen: a decoder-only language model whose norms come AFTER the sum — x <- norm1(alpha x + mixer(x)), x <- norm2(alpha x + ff(x)) —
and whose sublayers read their input h as h + conv(h), a short causal convolution over time on each channel.  Mixers: sliding-window
LATENT attention (queries through a normed latent, keys and values through another, one rotated key part shared by all heads, an
elementwise sigmoid gate on the concatenated heads), optionally on the latents of an earlier layer (kv_from); and causal grouped-query
attention without rotation, with per-head query / key norm, a learned temperature per head and a learned LOGARITHMIC distance bias
per head.  Feed-forward: a gelu-gated unit, or none.  This module only reads the checkpoint's config.json into the generic layer list
of leopard_b200/seqlm.py and names its tensors; the mechanisms themselves are the shared ones.

config.json keys: architecture, vocab, width, norm.eps, embedding.scale, postln_alpha, canon.taps, layers[] = {type: "latent_attention" |
"attention", mixer: {...}, mlp: null | {kind: "dense", ff}}.
  latent_attention mixer: heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot.{base, dims}, mask.size, kv_from (optional).
  attention mixer: heads, kv_heads, dim, vdim, scale.
Tensor names: embed, head, final.norm, and per layer l<i>.{norm1, norm2, canon1, canon2, mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o} |
mix.{q, k, v, q.norm, k.norm, temp, r1, r2, o}, mlp.{gate, up, down}}.
"""
from __future__ import annotations

import json
from pathlib import Path
from typing import Optional

from .safetensors_io import SafetensorsFile
from .seqlm import DenseFFConfig, LatentAttentionConfig, LayerConfig, RotaryConfig, SeqLMConfig, SeqLMEngine, SeqLMWeights, WindowAttentionConfig

ARCHITECTURE = "Komazen"
NO_ROTATION = RotaryConfig(dims=0, base=10000.0)
CONV_TENSORS = {"conv1": "canon1", "conv2": "canon2"}


def _window(m: dict) -> Optional[int]:
    size = (m.get("mask") or {}).get("size")
    return int(size) if size else None


def _mixer(kind: str, m: dict):
    heads, dim = int(m["heads"]), int(m["dim"])
    vdim = int(m.get("vdim", dim))
    if kind == "latent_attention":
        rot, rot_dim, kv_from = m.get("rot"), int(m["rot_dim"]), m.get("kv_from")
        return LatentAttentionConfig(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                                     rot=RotaryConfig(dims=int(rot["dims"]), base=float(rot["base"])) if rot and rot_dim else NO_ROTATION,
                                     window=_window(m), q_rank=int(m["q_rank"]), out_gate=True,
                                     kv_from=int(kv_from) if kv_from is not None else None)
    if kind == "attention":
        return WindowAttentionConfig(heads=heads, kv_heads=int(m.get("kv_heads", heads)), dim=dim, vdim=vdim, scale=float(m["scale"]),
                                     rot=NO_ROTATION, qk_norm="head", window=_window(m), head_temp=True, distance_bias=True)
    raise ValueError(f"unknown mixer type {kind!r}")


def _ff(f: Optional[dict]):
    if f is None:
        return None
    if f["kind"] == "dense":
        return DenseFFConfig(ff=int(f["ff"]), act="gelu_glu")
    raise ValueError(f"unknown feed-forward kind {f['kind']!r}")


def config_from_dict(d: dict) -> SeqLMConfig:
    if d.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config: architecture = {d.get('architecture')!r}")
    taps = int((d.get("canon") or {}).get("taps", 0))
    layers = tuple(LayerConfig(mixer=_mixer(l["type"], l["mixer"]), ff=_ff(l.get("mlp")), input_conv=taps) for l in d["layers"])
    return SeqLMConfig(architecture=ARCHITECTURE, vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]), layers=layers,
                       norm="post", post_alpha=float(d["postln_alpha"]), embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)))


def tensor_name(layer: Optional[int], key: str) -> str:
    return key if layer is None else f"l{layer}.{CONV_TENSORS.get(key, key)}"


def load(path, dtype: str = "bfloat16", device="cuda", lib=None, **engine_kw) -> SeqLMEngine:
    """A folder with config.json and model.safetensors -> an engine ready to step."""
    path = Path(path)
    cfg = config_from_dict(json.loads((path / "config.json").read_text()))
    st = SafetensorsFile(path / "model.safetensors")
    try:
        weights = SeqLMWeights(cfg, lambda n: st[n], tensor_name, device)
    finally:
        st.close()
    return SeqLMEngine(cfg, weights, dtype=dtype, lib=lib, **engine_kw)


def from_state_dict(d: dict, tensors: dict, dtype: str = "bfloat16", device="cuda", lib=None, **engine_kw) -> SeqLMEngine:
    """d: the parsed config.json; tensors: {checkpoint name: tensor}"""
    cfg = config_from_dict(d)
    return SeqLMEngine(cfg, SeqLMWeights(cfg, lambda n: tensors[n], tensor_name, device), dtype=dtype, lib=lib, **engine_kw)
