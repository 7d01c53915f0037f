"""Plain, slow float64 implementation of the Komazen layers: what the tests compare the post-norm layer form, the causal input
convolution, latent attention with query latents, shared latents and an elementwise output gate, grouped-query attention with a
temperature and a logarithmic distance bias per head, and the gelu-gated feed-forward of leopard_b200/seqlm.py with.  One function per
mechanism, whole sequences from position 0 only, nothing cached or cut, nothing shared with the product path: it takes the parsed
config.json and a {name: tensor} dict.

Notation: T tokens, D width, H query heads, G key / value heads (query head h reads group h // (H // G)), d key size, e value size.
"""
from __future__ import annotations

import math
from typing import Dict, Optional, Tuple

import torch

DT = torch.float64


def rms_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square (eps inside the root), times a plain gain"""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def with_convolution(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """h_t plus, per channel, the sum over the last K inputs (the current one last) weighted by w [D, K]; zeros before the start"""
    T, K = h.shape[0], w.shape[1]
    out = h.clone()
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def rotate(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """rows x [T, ..., n] at positions 0 .. T-1: pairs (i, i + dims/2) of the first `dims` entries turn by p * base^(-2i/dims)"""
    n = rot["dims"] // 2
    out = x.clone()
    for p in range(x.shape[0]):
        for i in range(n):
            a = p * rot["base"] ** (-2.0 * i / rot["dims"])
            u, v = x[p, ..., i], x[p, ..., i + n]
            out[p, ..., i] = u * math.cos(a) - v * math.sin(a)
            out[p, ..., i + n] = v * math.cos(a) + u * math.sin(a)
    return out


def visible(T: int, window: Optional[int]) -> torch.Tensor:
    """[T, T] bool: position i sees j <= i, with a window only the last `window` positions (itself among them)"""
    m = torch.zeros(T, T, dtype=torch.bool)
    for i in range(T):
        for j in range(i + 1):
            m[i, j] = window is None or i - j < window
    return m


def latents(h, w, p: str, m: dict, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """what a latent layer caches: the normed latent c [T, kv_rank] and the rotated key part all heads share [T, rot_dim]"""
    y = h @ w[p + "dkv"].T
    c = rms_norm(y[:, : m["kv_rank"]], w[p + "dkv.norm"], eps)
    return c, rotate(y[:, m["kv_rank"]:], m["rot"])


def latent_attention(h, w, p: str, m: dict, eps: float, shared=None):
    """softmax attention whose keys and values are up-projections of a latent; `shared`: another layer's (c, rotated key part).
    Returns (output [T, D], (c, rotated key part))"""
    T, H, d, r, e = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = shared if shared is not None else latents(h, w, p, m, eps)
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, d + r)
    qr = rotate(q[..., d:], m["rot"])
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, e)
    see = visible(T, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, e, dtype=DT)
    for hd in range(H):
        s = (q[:, hd, :d] @ k[:, hd].T + qr[:, hd] @ kr.T) * m["scale"]
        out[:, hd] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, hd]
    o = out.reshape(T, H * e) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T, (c, kr)


def biased_attention(h, w, p: str, m: dict, eps: float) -> torch.Tensor:
    """causal grouped-query attention without rotation: score q . k * scale * temp_h - r1_h ln(1 + r2_h (i - j))"""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w[p + "q"].T).view(T, H, d), w[p + "q.norm"], eps)
    k = rms_norm((h @ w[p + "k"].T).view(T, G, d), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T).view(T, G, e)
    i = torch.arange(T, dtype=DT)
    dist = (i[:, None] - i[None, :]).clamp(min=0)
    see = visible(T, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, e, dtype=DT)
    for hd in range(H):
        g = hd // (H // G)
        s = q[:, hd] @ k[:, g].T * m["scale"] * w[p + "temp"][hd] - w[p + "r1"][hd] * torch.log(1.0 + w[p + "r2"][hd] * dist)
        out[:, hd] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g]
    return out.reshape(T, H * e) @ w[p + "o"].T


def feed_forward(h, w, p: str) -> torch.Tensor:
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, taps: Optional[list] = None) -> torch.Tensor:
    """logits [T, vocab] of one whole sequence from position 0; taps (a list) receives the stream after every layer"""
    w = {k: v.to(DT) for k, v in w.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    cached = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = with_convolution(x, w[p + "canon1"])
        if layer["type"] == "latent_attention":
            j = m.get("kv_from")
            y, cached[i] = latent_attention(h, w, p + "mix.", m, eps, cached[j] if j is not None else None)
        elif layer["type"] == "attention":
            y = biased_attention(h, w, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = rms_norm(alpha * x + y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(with_convolution(x, w[p + "canon2"]), w, p + "mlp.")
            x = rms_norm(alpha * x + y, w[p + "norm2"], eps)
        if taps is not None:
            taps.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """bf16-representable random tensors under the checkpoint's names"""
    gen = torch.Generator().manual_seed(seed)
    D, K = cfg["width"], cfg["canon"]["taps"]
    out: Dict[str, torch.Tensor] = {}

    def mat(name, n, k, s=1.0):
        out[name] = (torch.randn(n, k, generator=gen) * s / math.sqrt(k)).to(torch.bfloat16).float()

    def vec(name, n, s=0.3, mean=1.0):
        out[name] = (torch.randn(n, generator=gen) * s + mean).to(torch.bfloat16).float()

    def positive(name, n, lo, hi):
        out[name] = (torch.rand(n, generator=gen) * (hi - lo) + lo).to(torch.bfloat16).float()

    mat("embed", cfg["vocab"], D, math.sqrt(D))
    mat("head", cfg["vocab"], D)
    vec("final.norm", D)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        mat(p + "canon1", D, K, 1.2)
        vec(p + "norm1", D)
        H, d, e = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "latent_attention":
            mat(q + "dq", m["q_rank"], D)
            vec(q + "dq.norm", m["q_rank"])
            mat(q + "uq", H * (d + m["rot_dim"]), m["q_rank"], 1.5)
            if m.get("kv_from") is None:
                mat(q + "dkv", m["kv_rank"] + m["rot_dim"], D)
                vec(q + "dkv.norm", m["kv_rank"])
            mat(q + "uk", H * d, m["kv_rank"], 1.5)
            mat(q + "uv", H * e, m["kv_rank"])
            mat(q + "g", H * e, D)
        else:
            mat(q + "q", H * d, D)
            mat(q + "k", m["kv_heads"] * d, D)
            mat(q + "v", m["kv_heads"] * e, D)
            vec(q + "q.norm", d)
            vec(q + "k.norm", d)
            positive(q + "temp", H, 0.6, 1.6)
            positive(q + "r1", H, 0.3, 1.5)
            positive(q + "r2", H, 0.1, 1.0)
        mat(q + "o", D, H * e, 2.0)
        f = layer.get("mlp")
        if f is not None:
            mat(p + "canon2", D, K, 1.2)
            vec(p + "norm2", D)
            mat(p + "mlp.gate", f["ff"], D, 1.5)
            mat(p + "mlp.up", f["ff"], D, 1.5)
            mat(p + "mlp.down", D, f["ff"], 2.0)
    return out
