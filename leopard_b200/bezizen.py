"""Bezizen: a decoder-only language model whose residual stream is kept as several copies joined by HYPER-CONNECTIONS (a sublayer reads a
learned sum of the copies, its result and a learned mixture of the old copies make the new ones), with learned positions added to a scaled
embedding.  Mixers: WKV time mixing (token-shifted projections, a matrix memory with a decay per key channel computed from the token, a
bonus for the current token); and a PARALLEL mixer of sliding-window attention — queries and keys through a short causal convolution, the
convolved keys serving as values, a linear distance bias, a query temperature that grows with the position, an elementwise output gate —
beside gated linear attention, the two outputs added with constant scales.  Feed-forward: a mixture of experts chosen by softmax scores
within the best groups, plus a shared expert, or none.  This module only reads the checkpoint's config.json into the generic layer list of
leopard_b200/seqlm.py and names its tensors; the mechanisms themselves are the shared ones.

config.json keys: architecture, vocab, width, max_positions, streams, norm.eps, embedding.scale, logit_scale, layers[] = {type: "wkv" |
"parallel", mixer: {...}, mlp: null | {kind: "moe", expert.ff, router.{experts, top, scale, groups.{count, keep}}, shared.ff (optional)}}.
  wkv mixer: heads, dim.
  parallel mixer: left = {heads, kv_heads, dim, vdim, scale, conv, mask.size, q_temp.{coef, every}}, right = {heads, dim, vdim, tau},
  left_scale, right_scale.
Tensor names: embed, pos, head, final.norm, and per layer l<i>.{norm1, norm2, hc1.{in, mix, out}, hc2.{in, mix, out}, mix.{mu.{r, k, v, g, w}, r,
k, v, g, w1, w2, w0, u, norm, o} | mix.left.{q, k, q.conv, k.conv, g, o}, mix.right.{q, k, v, g, a1, a2, a2.b, norm, o},
mlp.{router, e<j>.{gate, up, down}, shared.{gate, up, down}}}.
"""
from __future__ import annotations

import json
from pathlib import Path
from typing import Optional

from .safetensors_io import SafetensorsFile
from .seqlm import (GatedLinearConfig, LayerConfig, MoEConfig, ParallelMixerConfig, RotaryConfig, SeqLMConfig, SeqLMEngine, SeqLMWeights,
                    WindowAttentionConfig, WKVConfig)

ARCHITECTURE = "Bezizen"
NO_ROTATION = RotaryConfig(dims=0, base=10000.0)


def _attention(m: dict) -> WindowAttentionConfig:
    heads, dim = int(m["heads"]), int(m["dim"])
    size, temp = (m.get("mask") or {}).get("size"), m.get("q_temp")
    if int(m.get("vdim", dim)) != dim:
        raise ValueError(f"the keys are the values: dim = {dim} and vdim = {m['vdim']} must agree")
    return WindowAttentionConfig(heads=heads, kv_heads=int(m.get("kv_heads", heads)), dim=dim, vdim=dim, scale=float(m["scale"]), rot=NO_ROTATION,
                                 window=int(size) if size else None, qk_conv=int(m.get("conv") or 0), values_are_keys=True, distance_slope=True,
                                 pos_temp=(float(temp["coef"]), int(temp["every"])) if temp else None, out_gate=True)


def _mixer(kind: str, m: dict):
    if kind == "wkv":
        return WKVConfig(heads=int(m["heads"]), dim=int(m["dim"]))
    if kind == "parallel":
        r = m["right"]
        right = GatedLinearConfig(heads=int(r["heads"]), dim=int(r["dim"]), vdim=int(r.get("vdim", r["dim"])), tau=float(r["tau"]))
        return ParallelMixerConfig(left=_attention(m["left"]), right=right, scales=(float(m["left_scale"]), float(m["right_scale"])))
    raise ValueError(f"unknown mixer type {kind!r}")


def _ff(f: Optional[dict]):
    if f is None:
        return None
    if f["kind"] == "moe":
        r, sh = f["router"], f.get("shared")
        g = r.get("groups") or {"count": 1, "keep": 1}
        return MoEConfig(experts=int(r["experts"]), top=int(r["top"]), expert_ff=int(f["expert"]["ff"]), n_groups=int(g["count"]),
                         keep_groups=int(g["keep"]), router="group_softmax", weight_scale=float(r.get("scale", 1.0)),
                         shared_ff=int(sh["ff"]) if sh else 0, shared_gate=False)
    raise ValueError(f"unknown feed-forward kind {f['kind']!r}")


def config_from_dict(d: dict) -> SeqLMConfig:
    if d.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config: architecture = {d.get('architecture')!r}")
    layers = tuple(LayerConfig(mixer=_mixer(l["type"], l["mixer"]), ff=_ff(l.get("mlp"))) for l in d["layers"])
    return SeqLMConfig(architecture=ARCHITECTURE, vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]), layers=layers,
                       norm="pre_plain", streams=int(d["streams"]), learned_positions=int(d["max_positions"]),
                       embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)), logit_scale=float(d.get("logit_scale", 1.0)))


def tensor_name(layer: Optional[int], key: str) -> str:
    return key if layer is None else f"l{layer}.{key}"


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
