"""Plain, slow float64 implementation of the Bezizen layers: what the tests compare the hyper-connected streams, learned positions, the
WKV time mixing, gated linear attention, grouped-query attention whose values are its convolved keys, and the softmax router over groups
of experts of leopard_b200/seqlm.py with.  One function per mechanism, whole sequences from position 0 only, nothing cached or cut, nothing
shared with the product path: it takes the parsed config.json and a {name: tensor} dict.

Notation: T tokens, D width, H query heads, G key / value heads (query head h reads group h // (H // G)), d key size, e value size.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

DT = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square, eps inside the root"""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """per channel the weighted sum of the last K inputs, the current one under the last tap; zeros before the start.  u [T, C], w [C, K]"""
    T, K = u.shape[0], w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                out[t] += w[:, j] * u[s]
    return out


def previous(h: torch.Tensor) -> torch.Tensor:
    """the row before each row; zeros before the first"""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)


def decayed_memory(q, k, v, decay, bonus: Optional[torch.Tensor] = None) -> torch.Tensor:
    """one head's matrix memory S [d, e], S_t = diag(decay_t) S_(t-1) + k_t v_t^T from zero.  Without a bonus the query reads S_t; with
    one it reads S_(t-1) + diag(bonus) k_t v_t^T.  q, k, decay [T, d], v [T, e] -> [T, e]"""
    T, d, e = q.shape[0], k.shape[1], v.shape[1]
    S = torch.zeros(d, e, dtype=DT)
    out = torch.zeros(T, e, dtype=DT)
    for t in range(T):
        now = torch.outer(k[t], v[t])
        if bonus is not None:
            out[t] = (S + bonus[:, None] * now).T @ q[t]
        S = decay[t][:, None] * S + now
        if bonus is None:
            out[t] = S.T @ q[t]
    return out


def wkv_mixer(h, w, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, d = h.shape[0], m["heads"], m["dim"]
    step = previous(h) - h
    mixed = {s: h + step * w[p + "mu." + s] for s in "rkvgw"}
    r, k, v = ((mixed[s] @ w[p + s].T).view(T, H, d) for s in "rkv")
    gate = silu(mixed["g"] @ w[p + "g"].T)
    z = torch.tanh(mixed["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = torch.exp(-torch.exp(z)).view(T, H, d)
    o = torch.stack([decayed_memory(r[:, i], k[:, i], v[:, i], decay[:, i], w[p + "u"][i]) for i in range(H)], 1)
    return (rms(o, eps).reshape(T, H * d) * w[p + "norm"] * gate) @ w[p + "o"].T


def gated_linear_attention(h, w, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, e)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    decay = (torch.sigmoid(z) ** (1.0 / m["tau"])).view(T, H, d)
    o = torch.stack([decayed_memory(q[:, i], k[:, i], v[:, i], decay[:, i]) for i in range(H)], 1)
    o = rms(o, eps) * w[p + "norm"]
    return (o.reshape(T, H * e) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def visible(T: int, window: Optional[int]) -> torch.Tensor:
    """[T, T] bool: position i sees j <= i, with a window only the last `window` positions (itself among them)"""
    m = torch.zeros(T, T, dtype=torch.bool)
    for i in range(T):
        for j in range(i + 1):
            m[i, j] = window is None or i - j < window
    return m


def sloped_attention(h, w, p: str, m: dict) -> torch.Tensor:
    """softmax attention on convolved queries and keys, the keys serving as values; queries grow with the logarithm of their position,
    scores fall linearly with the distance, the heads' outputs are gated"""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = causal_conv(h @ w[p + "q"].T, w[p + "q.conv"]).view(T, H, d)
    k = causal_conv(h @ w[p + "k"].T, w[p + "k.conv"]).view(T, G, d)
    see = visible(T, (m.get("mask") or {}).get("size"))
    temp = torch.tensor([1.0 + m["q_temp"]["coef"] * math.log((i + 1) // m["q_temp"]["every"] + 1) for i in range(T)], dtype=DT)
    pos = torch.arange(T, dtype=DT)
    out = torch.zeros(T, H, d, dtype=DT)
    for i in range(H):
        kk = k[:, i // (H // G)]
        s = (q[:, i] * temp[:, None]) @ kk.T * m["scale"] - 2.0 ** (-8.0 * (i + 1) / H) * (pos[:, None] - pos[None, :])
        out[:, i] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ kk
    return (out.reshape(T, H * d) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def unit(h, w, p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p: str, r: dict) -> List[Dict[int, float]]:
    """per token {expert: weight}: softmax scores, the experts of the groups with the largest best score, the largest of those, their
    scores over their sum, times a constant"""
    s = torch.softmax(h @ w[p + "router"].T, -1)
    g = r.get("groups") or {"count": 1, "keep": 1}
    size = r["experts"] // g["count"]
    out = []
    for row in s.tolist():
        best = sorted(range(g["count"]), key=lambda i: -max(row[i * size:(i + 1) * size]))[: g["keep"]]
        pick = sorted((e for i in best for e in range(i * size, (i + 1) * size)), key=lambda e: -row[e])[: r["top"]]
        total = sum(row[e] for e in pick) + 1e-20
        out.append({e: row[e] / total * r.get("scale", 1.0) for e in pick})
    return out


def experts(h, w, p: str, f: dict) -> torch.Tensor:
    out = torch.zeros_like(h)
    for t, choice in enumerate(route(h, w, p, f["router"])):
        for e, weight in choice.items():
            out[t] += weight * unit(h[t], w, f"{p}e{e}.")
    return out + unit(h, w, p + "shared.") if f.get("shared") else out


def through_streams(xs: torch.Tensor, w, p: str, sublayer) -> torch.Tensor:
    """xs [S, T, D]: the sublayer reads sum_s in[s] x_s, and every stream becomes a mixture of all old ones plus its share of the result"""
    y = sublayer(torch.einsum("s,std->td", w[p + "in"], xs))
    return torch.einsum("st,sij->tij", w[p + "mix"], xs) + w[p + "out"][:, None, None] * y


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, taps: Optional[list] = None) -> torch.Tensor:
    """logits [T, vocab] of one whole sequence from position 0; taps (a list) receives the sum of the streams after every layer"""
    w = {k: v.to(DT) for k, v in w.items()}
    eps, T = cfg["norm"]["eps"], len(tokens)
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"] + w["pos"][:T]
    xs = torch.stack([x] * cfg["streams"], 0)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]

        def mixer(u):
            h = rms(u, eps) * w[p + "norm1"]
            if layer["type"] == "wkv":
                return wkv_mixer(h, w, p + "mix.", m, eps)
            if layer["type"] == "parallel":
                return (m["left_scale"] * sloped_attention(h, w, p + "mix.left.", m["left"])
                        + m["right_scale"] * gated_linear_attention(h, w, p + "mix.right.", m["right"], eps))
            raise ValueError(layer["type"])
        xs = through_streams(xs, w, p + "hc1.", mixer)
        if layer.get("mlp") is not None:
            xs = through_streams(xs, w, p + "hc2.", lambda u: experts(rms(u, eps) * w[p + "norm2"], w, p + "mlp.", layer["mlp"]))
        if taps is not None:
            taps.append(xs.sum(0))
    return (rms(xs.sum(0), eps) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"]


def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """bf16-representable random tensors under the checkpoint's names"""
    gen = torch.Generator().manual_seed(seed)
    D, S = cfg["width"], cfg["streams"]
    out: Dict[str, torch.Tensor] = {}

    def mat(name, *shape, s=1.0):
        out[name] = (torch.randn(*shape, generator=gen) * s / math.sqrt(shape[-1])).to(torch.bfloat16).float()

    def vec(name, *shape, s=0.3, mean=1.0):
        out[name] = (torch.randn(*shape, generator=gen) * s + mean).to(torch.bfloat16).float()

    def hyper(p):
        vec(p + "in", S, mean=1.0 / S)
        vec(p + "out", S, s=0.4)
        out[p + "mix"] = (0.8 * torch.eye(S) + 0.2 * torch.randn(S, S, generator=gen)).to(torch.bfloat16).float()

    mat("embed", cfg["vocab"], D, s=math.sqrt(D))
    mat("pos", cfg["max_positions"], D, s=math.sqrt(D))
    mat("head", cfg["vocab"], D)
    vec("final.norm", D)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        vec(p + "norm1", D)
        hyper(p + "hc1.")
        q = p + "mix."
        if layer["type"] == "wkv":
            n, rank = m["heads"] * m["dim"], m.get("rank", 5)      # a checkpoint gives the rank by the shapes of w1 and w2
            for s in "rkvgw":
                out[q + "mu." + s] = torch.rand(D, generator=gen).to(torch.bfloat16).float()
            for s in "rkvg":
                mat(q + s, n, D, s=1.3)
            mat(q + "w1", rank, D)
            mat(q + "w2", n, rank, s=1.5)
            vec(q + "w0", n, s=0.8, mean=-1.0)
            vec(q + "u", m["heads"], m["dim"], s=0.7, mean=0.5)
            vec(q + "norm", n)
            mat(q + "o", D, n, s=2.0)
        else:
            l, r = m["left"], m["right"]
            nq, nk = l["heads"] * l["dim"], l["kv_heads"] * l["dim"]
            mat(q + "left.q", nq, D, s=1.5)
            mat(q + "left.k", nk, D, s=1.5)
            mat(q + "left.q.conv", nq, l["conv"], s=1.3)
            mat(q + "left.k.conv", nk, l["conv"], s=1.3)
            mat(q + "left.g", nq, D)
            mat(q + "left.o", D, nq, s=2.0)
            n, e, rank = r["heads"] * r["dim"], r["heads"] * r["vdim"], r.get("rank", 3)
            mat(q + "right.q", n, D)
            mat(q + "right.k", n, D)
            mat(q + "right.v", e, D)
            mat(q + "right.g", e, D)
            mat(q + "right.o", D, e, s=2.0)
            vec(q + "right.norm", r["vdim"])
            mat(q + "right.a1", rank, D)
            mat(q + "right.a2", n, rank, s=2.0)
            vec(q + "right.a2.b", n, s=1.0, mean=0.5)
        f = layer.get("mlp")
        if f is not None:
            vec(p + "norm2", D)
            hyper(p + "hc2.")
            mat(p + "mlp.router", f["router"]["experts"], D, s=2.0)
            parts = [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + ([("shared", f["shared"]["ff"])] if f.get("shared") else [])
            for name, ff in parts:
                mat(f"{p}mlp.{name}.gate", ff, D, s=1.5)
                mat(f"{p}mlp.{name}.up", ff, D, s=1.5)
                mat(f"{p}mlp.{name}.down", D, ff, s=2.0)
    return out
