"""Bezizen on the step engine against the plain implementation (oracle/bezizen.py): every mechanism alone, whole prompts against
token-by-token decoding, prompts cut into portions down to one and two tokens (fewer than the convolution looks back) and up to several
pieces of the recurrence, batches of unequal requests, pages and slots that are given back and taken again, keys just inside and just
outside a window (in a prompt and decoded), page borders, a first token that the memories still hold at the end, the first tokens of a
sequence, long decoding, sizes that happen to be equal or one, both precisions, and greedy generation through the scheduler and the
command line.  Where random weights would hide a fault, the configuration's score scale is raised so that every softmax leans on few keys,
or the decays are set so that one token stands out, and the test first shows on the oracle itself that the fault would be noticed.  On the
kernel sources under the CPU emulator and, marked gpu, on the native library."""
import copy
import ctypes as C
import json
import math

import pytest
import torch

from leopard_b200 import bezizen
from leopard_b200.scheduler import Request, Scheduler, generate
from leopard_b200.seqlm import StepEntry
from oracle import bezizen as O
from bezizen_common import TOL, backend, emu_lib, make_engine, mixed_model, model, moe, parallel_layer, rel_err, wkv_layer  # noqa: F401


def _tokens(n, vocab, seed=0):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def _all(n):
    return list(range(n))


def _rows(got, want):
    """relative error of every row"""
    got, want = got.double().cpu(), want.double()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()


def _prompt_then_decode(eng, toks, n_prompt, key="r"):
    got = [eng.step([StepEntry(key, toks[:n_prompt], _all(n_prompt))])]
    for t in toks[n_prompt:]:
        got.append(eng.step([StepEntry(key, [t], [0])]))
    return torch.cat(got, 0)


MODELS = {
    "wkv": ([wkv_layer()], {}),
    "wkv, odd sizes, one head": ([wkv_layer(heads=1, dim=19, rank=1)], {"width": 11, "streams": 1}),
    "wkv, heads of several warps and column groups": ([wkv_layer(heads=2, dim=40, rank=9)], {"streams": 4}),
    "wkv + experts": ([wkv_layer(mlp=moe())], {}),
    "parallel": ([parallel_layer()], {}),
    "parallel, one key head, long convolution": ([parallel_layer(heads=3, kv_heads=1, dim=6, conv=6, window=3, gheads=1, gdim=18, gvdim=35)],
                                                 {"streams": 5, "width": 13}),
    "parallel, every head its own keys, one tap": ([parallel_layer(heads=2, kv_heads=2, dim=16, conv=1, gheads=2, gdim=3, gvdim=70)], {"streams": 1}),
    "parallel, wide value heads": ([parallel_layer(gheads=1, gdim=5, gvdim=140)], {}),
    "parallel + experts": ([parallel_layer(mlp=moe(experts=5, top=3, groups=None, shared=0))], {"streams": 3, "width": 16}),
}


@pytest.mark.parametrize("name", list(MODELS))
def test_each_mechanism_alone(backend, name):
    """a small model: the whole prompt in one step, and the same tokens with the last ones decoded through cache and state"""
    layers, kw = MODELS[name]
    cfg = model(layers, **kw)
    w = O.random_weights(cfg, seed=3)
    toks = _tokens(9, cfg["vocab"], seed=1)
    res = []
    want = O.forward(cfg, w, toks, taps=res)
    eng = make_engine(cfg, w, backend)
    taps = []
    eng.tap = lambda li, x: taps.append(x.clone())
    got = eng.step([StepEntry("p", toks, _all(9))])
    assert len(taps) == len(res)
    for a, b in zip(taps, res):                                   # the sum of the streams after every layer
        assert rel_err(a, b) < TOL["float32"]
    assert float(_rows(got, want).max()) < 5 * TOL["float32"]
    eng.tap = None
    eng.finish("p")
    assert float(_rows(_prompt_then_decode(eng, toks, 5), want).max()) < 5 * TOL["float32"]


def test_every_piece_matters_on_the_oracle():
    """each piece, shown to move the logits when it is left out or changed"""
    cfg = mixed_model()
    w = O.random_weights(cfg, seed=4)
    toks = _tokens(12, cfg["vocab"], seed=5)
    want = O.forward(cfg, w, toks)
    changes = {"pos": 0.0, "l0.mix.mu.r": 0.0, "l0.mix.mu.k": 0.0, "l0.mix.mu.v": 0.0, "l0.mix.mu.g": 0.0, "l0.mix.mu.w": 0.0, "l0.mix.w0": -1.0,
               "l0.mix.w2": 0.0, "l0.mix.u": 1.0, "l0.mix.norm": 1.0, "l2.mix.u": 0.0, "l1.mix.left.q.conv": 0.5, "l1.mix.left.k.conv": 0.5,
               "l1.mix.left.g": 0.0, "l1.mix.right.a2": 0.0, "l1.mix.right.a2.b": 0.0, "l1.mix.right.norm": 1.0, "l1.mix.right.g": 0.01,
               "l0.hc2.in": 0.5, "l1.hc1.in": 0.5, "l0.hc2.out": 1.0, "l1.hc1.mix": 0.3, "l2.hc1.mix": 0.3, "l0.norm2": 1.0, "l0.mlp.router": 0.0,
               "l0.mlp.shared.gate": 0.0, "final.norm": 1.0}
    for name, value in changes.items():
        w2 = dict(w)
        w2[name] = torch.full_like(w[name], value)
        assert float(_rows(O.forward(cfg, w2, toks), want).median()) > 100 * TOL["float32"], name
    for path, value in ((("logit_scale",), 0.7), (("embedding", "scale"), 1.4), (("norm", "eps"), 1e-2), (("layers", 1, "mixer", "left_scale"), 1.1),
                        (("layers", 1, "mixer", "right_scale"), 0.8), (("layers", 1, "mixer", "left", "scale"), 0.55),
                        (("layers", 1, "mixer", "left", "q_temp", "coef"), 0.3), (("layers", 1, "mixer", "left", "q_temp", "every"), 2),
                        (("layers", 1, "mixer", "right", "tau"), 5.0), (("layers", 0, "mlp", "router", "scale"), 1.5)):
        c2 = copy.deepcopy(cfg)
        node = c2
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        assert float(_rows(O.forward(c2, w, toks), want).median()) > 20 * TOL["float32"], path
    c2 = copy.deepcopy(cfg)
    c2["layers"][0]["mlp"]["router"]["groups"]["keep"] = 3      # some token's choice hangs on the groups
    assert float(_rows(O.forward(c2, w, toks), want).max()) > 1000 * TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_then_long_decoding(backend, dtype):
    """a prompt, then tokens one by one: windows pass over decoded tokens, pages fill up, the query temperature climbs, carried inputs
    and memories move on"""
    cfg = mixed_model()
    w = O.random_weights(cfg, seed=11)
    toks = _tokens(80, cfg["vocab"], seed=2)
    want = O.forward(cfg, w, toks)
    eng = make_engine(cfg, w, backend, dtype, max_tokens=96)
    got = _prompt_then_decode(eng, toks, 21)
    assert rel_err(got, want) < TOL[dtype]
    if dtype == "float32":
        assert float(_rows(got, want).max()) < 5 * TOL[dtype]


@pytest.mark.parametrize("cuts", [(2, 2, 3, 2), (1, 2, 8), (5, 66, 2, 101, 3)])
def test_portions_of_a_prompt(backend, cuts):
    """a prompt fed in portions, some shorter than the convolution looks back (5 taps), some so long that the recurrences run in pieces"""
    cfg = model([wkv_layer(mlp=moe()), parallel_layer(conv=5, window=7)])
    w = O.random_weights(cfg, seed=12)
    toks = _tokens(sum(cuts), cfg["vocab"], seed=3)
    want = O.forward(cfg, w, toks)
    eng = make_engine(cfg, w, backend, max_tokens=96)
    got, at = [], 0
    for n in cuts:
        got.append(eng.step([StepEntry("r", toks[at:at + n], _all(n))]))
        at += n
    assert float(_rows(torch.cat(got, 0), want).max()) < 5 * TOL["float32"]


def test_batch_of_unequal_requests_and_reuse(backend):
    """three requests of different lengths in one batch, decoded together while the short ones end; then a new request takes the
    pages and the slot that were given back (the pools are sized so that it must), whose carried inputs and memories it must not see"""
    cfg = mixed_model()
    w = O.random_weights(cfg, seed=13)
    lens = {"a": (1, 2), "b": (5, 3), "c": (70, 1)}            # prompt length, decoded tokens
    toks = {k: _tokens(p + d, cfg["vocab"], seed=30 + i) for i, (k, (p, d)) in enumerate(lens.items())}
    want = {k: O.forward(cfg, w, toks[k]) for k in lens}
    eng = make_engine(cfg, w, backend, max_tokens=80, max_seqs=3)
    got = {k: [] for k in lens}
    out = eng.step([StepEntry(k, toks[k][:p], [p - 1]) for k, (p, d) in lens.items()])
    for i, k in enumerate(lens):
        got[k].append(out[i:i + 1])
    live = list(lens)
    for step in range(3):
        live = [k for k in live if step < lens[k][1]]
        out = eng.step([StepEntry(k, [toks[k][lens[k][0] + step]], [0]) for k in live])
        for i, k in enumerate(live):
            got[k].append(out[i:i + 1])
        for k in live:
            if step + 1 == lens[k][1]:
                eng.finish(k)
    for k, (p, d) in lens.items():
        assert float(_rows(torch.cat(got[k], 0), want[k][p - 1:]).max()) < 5 * TOL["float32"], k
    c = eng.cache
    assert c.pages_in_use() == 0 and len(c.free_slots) == c.n_slots
    before = (c.n_slots, c.n_pages)
    t2 = _tokens(6, cfg["vocab"], seed=77)
    again = eng.step([StepEntry("a", t2, _all(6))])           # the name of an ended request, a used slot, used pages
    assert float(_rows(again, O.forward(cfg, w, t2)).max()) < 5 * TOL["float32"]
    eng.finish("a")
    one = eng.step([StepEntry("a", t2[:1], [0])])             # a first token that runs as a one-token step on a used slot
    two = eng.step([StepEntry("a", t2[1:2], [0])])
    assert float(_rows(torch.cat([one, two], 0), O.forward(cfg, w, t2[:2])).max()) < 5 * TOL["float32"]
    assert (c.n_slots, c.n_pages) == before


def _one_off(cfg, delta):
    c = copy.deepcopy(cfg)
    for l in c["layers"]:
        if l["type"] == "parallel":
            l["mixer"]["left"]["mask"]["size"] += delta
    return c


@pytest.mark.parametrize("mode", ["prompt", "decoded"])
def test_edge_of_the_window(backend, mode):
    """many heads, whose last slopes are nearly flat, and a large score scale make the softmaxes lean on few keys wherever they are: the
    oracle with a window one token longer or shorter differs by far more than the tolerance on many rows, and the engine agrees with the
    right one, across page borders (pages of 4 tokens), with the pages behind the window given back while the request runs"""
    cfg = model([parallel_layer(heads=8, kv_heads=4, dim=4, window=6, scale=2.0)])
    w = O.random_weights(cfg, seed=21)
    toks = _tokens(41, cfg["vocab"], seed=6)
    want = O.forward(cfg, w, toks)
    for delta in (-1, 1):
        off = _rows(O.forward(_one_off(cfg, delta), w, toks), want)
        edge = 6 + min(delta, 0)
        assert int((off[edge:] > 200 * TOL["float32"]).sum()) >= 8
        assert float(off[:edge].max()) < 1e-12                      # rows that see the same either way
    eng = make_engine(cfg, w, backend, max_tokens=8)
    got = eng.step([StepEntry("r", toks, _all(41))]) if mode == "prompt" else _prompt_then_decode(eng, toks, 3)
    assert float(_rows(got, want).max()) < 5 * TOL["float32"]
    assert sum(p >= 0 for p in eng.cache.get("r").pages) <= 3      # only the pages of the window are still held


@pytest.mark.parametrize("kind", ["wkv", "gated"])
def test_the_first_token_is_remembered(backend, kind):
    """decays close to one: the oracle with another first token differs at the end of a prompt of several pieces and after it, and the engine
    agrees with the right one; the slot holds the state between the portions"""
    if kind == "wkv":
        cfg = model([wkv_layer(heads=1, dim=8)])
    else:
        cfg = model([parallel_layer(window=2, gheads=1, gdim=8, gvdim=6, tau=64.0)])
    w = O.random_weights(cfg, seed=25)
    if kind == "wkv":
        w["l0.mix.w0"] = w["l0.mix.w0"] - 6.0
    w["pos"] = w["pos"] * 0.25
    toks = _tokens(130, cfg["vocab"], seed=26)
    want = O.forward(cfg, w, toks)
    other = O.forward(cfg, w, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    assert int((_rows(other[-10:], want[-10:]) > 50 * TOL["float32"]).sum()) >= 5
    eng = make_engine(cfg, w, backend, max_tokens=8)
    got = [eng.step([StepEntry("r", toks[:97], _all(97))]), eng.step([StepEntry("r", toks[97:126], _all(29))])]
    got += [eng.step([StepEntry("r", [t], [0])]) for t in toks[126:]]
    assert float(_rows(torch.cat(got, 0), want).max()) < 5 * TOL["float32"]


@pytest.mark.gpu
def test_far_keys_and_edges_among_hundreds():
    """windows of hundreds of keys (several key tiles, many pages), sharp softmaxes, long memories: the oracle with a window one token off
    and a changed first token is told apart; portions start at every kind of offset and the end is decoded"""
    layers = [parallel_layer(heads=16, kv_heads=4, dim=8, conv=4, window=150, scale=0.9, every=40, gheads=4, gdim=20, gvdim=24, tau=30.0),
              wkv_layer(heads=3, dim=24, rank=8, mlp=moe()),
              parallel_layer(heads=16, kv_heads=16, dim=8, conv=2, window=131, scale=0.9, every=64, gheads=2, gdim=16, gvdim=130, tau=30.0)]
    cfg = model(layers, width=24, positions=400)
    w = O.random_weights(cfg, seed=31)
    w["l1.mix.w0"] = w["l1.mix.w0"] - 4.0
    toks = _tokens(330, cfg["vocab"], seed=32)
    want = O.forward(cfg, w, toks)
    for delta in (-1, 1):
        off = _rows(O.forward(_one_off(cfg, delta), w, toks), want)
        assert int((off[150:] > 200 * TOL["float32"]).sum()) >= 15
    first = O.forward(cfg, w, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    assert int((_rows(first[-100:], want[-100:]) > 20 * TOL["float32"]).sum()) >= 50
    eng = make_engine(cfg, w, ("cuda", None), max_tokens=400, page_size=16)
    got, at = [], 0
    for n in (129, 2, 67, 101, 3):
        got.append(eng.step([StepEntry("r", toks[at:at + n], _all(n))]))
        at += n
    for t in toks[at:]:
        got.append(eng.step([StepEntry("r", [t], [0])]))
    assert float(_rows(torch.cat(got, 0), want).max()) < 5 * TOL["float32"]
    # the same tokens in a batch with a short request, in the serving precision, against themselves alone
    half = make_engine(cfg, w, ("cuda", None), "bfloat16", max_tokens=800, page_size=16)
    both = half.step([StepEntry("x", toks[:7], [6]), StepEntry("y", toks[:300], _all(300))])
    alone = half.step([StepEntry("z", toks[:300], _all(300))])
    assert rel_err(both[1:], want[:300]) < 2 * TOL["bfloat16"] and rel_err(both[1:], alone) < 5e-3


@pytest.mark.gpu
def test_wide_layers_on_the_tensor_cores():
    """sizes at which the serving precision sends its products to the tcgen05 GEMM: the five operands of the time mixing, the padded
    low-rank projection and its split second product, both branches of the parallel mixer, experts"""
    layers = [wkv_layer(heads=4, dim=64, rank=32, mlp=moe(experts=4, top=2, groups=(2, 1), ff=64, shared=128)),
              parallel_layer(heads=8, kv_heads=4, dim=32, conv=4, window=100, scale=0.2, every=50, gheads=4, gdim=48, gvdim=64, rank=36, tau=16.0),
              wkv_layer(heads=2, dim=128, rank=40, mlp=moe(experts=4, top=1, groups=None, ff=128, shared=0))]
    plain = copy.deepcopy(layers)
    for l in plain:
        l["mlp"] = None
    toks = _tokens(300, 300, seed=42)
    for experts, ls in ((False, plain), (True, layers)):
        cfg = model(ls, width=128, vocab=300, positions=512)
        w = O.random_weights(cfg, seed=41)
        want = O.forward(cfg, w, toks)
        for dtype in ("float32", "bfloat16"):
            eng = make_engine(cfg, w, ("cuda", None), dtype, max_tokens=512, page_size=64)
            got = [eng.step([StepEntry("r", toks[:280], _all(280))])]
            got += [eng.step([StepEntry("r", [t], [0])]) for t in toks[280:]]
            off = _rows(torch.cat(got, 0), want)
            # rounded operands may turn a close call of a router: with experts the serving precision is judged by the typical row
            assert float(off.median()) < TOL[dtype], (experts, dtype)
            if not experts or dtype == "float32":
                assert float(off.max()) < 5 * TOL[dtype], (experts, dtype)


# ---------------------------------------------------------------------------------------------------------------- kernels
def _bare_engine(backend, width=8, **kw):
    """an engine whose helpers and batch tables the kernel tests borrow"""
    cfg = model([wkv_layer(heads=1, dim=4)], width=width)
    return make_engine(cfg, O.random_weights(cfg, seed=1), backend, **kw)


@pytest.mark.parametrize("dim, vdim, bonus, lens", [(6, 5, True, (3, 1)), (17, 33, False, (71, 5)), (64, 64, True, (100, 70)), (40, 129, False, (66, 2)),
                                                    (130, 100, True, (5, 4)), (256, 20, False, (2, 67))])
def test_decayed_memory_kernel(backend, dim, vdim, bonus, lens):
    """the recurrence alone, two requests of unequal length: every column width, one and several warps, pieces and whole requests, decays
    from practically zero to practically one; then the state left in the slots carries on, once more as a portion and once as one-token
    steps whose decays are made from their low-rank factors.  Slots start with rubbish."""
    from leopard_b200 import _lib
    from leopard_b200.seqlm import _Batch
    H, rank = 2, 3
    eng = _bare_engine(backend, max_tokens=256)
    dev, L = eng.device, eng.L
    g = torch.Generator().manual_seed(dim)
    total = {"a": lens[0] + 4, "b": lens[1] + 4}
    data, want = {}, {}
    w2 = torch.randn(H * dim, rank, generator=g).to(torch.bfloat16)
    zb = torch.randn(H * dim, generator=g)
    u = torch.randn(H, dim, generator=g)
    gain = torch.rand(H * vdim, generator=g) + 0.5
    for k, n in total.items():
        r = {"q": torch.randn(n, H * dim, generator=g), "k": torch.randn(n, H * dim, generator=g), "v": torch.randn(n, H * vdim, generator=g),
             "g": torch.randn(n, H * vdim, generator=g), "t": 2.5 * torch.randn(n, rank, generator=g)}
        act = torch.tanh(r["t"].double()) if bonus else r["t"].double()
        z = act @ w2.double().T + zb.double()
        z[:, ::7] = -12.0 if bonus else 12.0                      # channels that forget nothing
        z[1::3, 1::5] = 5.0 if bonus else -60.0                   # and now and then everything
        a = torch.exp(-torch.exp(z)) if bonus else torch.sigmoid(z) ** 0.25
        r["z"] = z.float()
        heads = []
        for h in range(H):
            s, e = slice(h * dim, (h + 1) * dim), slice(h * vdim, (h + 1) * vdim)
            o = O.decayed_memory(0.3 * r["q"][:, s].double(), r["k"][:, s].double(), r["v"][:, e].double(), a[:, s], u[h].double() if bonus else None)
            heads.append(O.rms(o, 1e-5) * gain[h * vdim:(h + 1) * vdim].double())
        data[k], want[k] = r, torch.cat(heads, 1) * O.silu(r["g"].double())
    state = torch.full((2, H, dim, vdim), float("nan"), device=dev)
    gain_d, u_d, w2_d, zb_d = gain.to(dev), u.reshape(-1).contiguous().to(dev), w2.to(dev), zb.to(dev)

    def run(rows):
        b = _Batch(eng, [StepEntry(k, [0] * n) for k, n in rows.items()])
        at = {k: eng.cache.get(k).length for k in rows}
        cat = {f: torch.cat([data[k][f][at[k]:at[k] + n] for k, n in rows.items()], 0).to(dev) for f in "qkvgtz"}
        out = torch.full((b.R, H * vdim), float("nan"), device=dev)
        d = _lib.GlaDesc(q=_lib.ptr(cat["q"]), k=_lib.ptr(cat["k"]), v=_lib.ptr(cat["v"]), ldq=H * dim, ldk=H * dim, ldv=H * vdim, heads=H, dim=dim,
                         vdim=vdim, q_scale=0.3, decay=_lib.GLA_DECAY_DOUBLE_EXP if bonus else _lib.GLA_DECAY_SIGMOID_POW, decay_exp=0.25,
                         z=_lib.ptr(cat["z"]), ldz=H * dim, bonus=_lib.ptr(u_d) if bonus else None, out_gain=_lib.ptr(gain_d), gain_stride=vdim,
                         gate=_lib.ptr(cat["g"]), ldg=H * vdim, eps=1e-5, state=_lib.ptr(state), slot_stride=state.stride(0), out=_lib.ptr(out),
                         ldo=H * vdim, out_fp32=1)
        n_ws = int(L.lp_gla_workspace_bytes(b.n_chunks, b.R, max(b.lens), H, dim, vdim))
        ws = torch.full((n_ws // 4 + 1,), float("nan"), device=dev)
        rc = L.lp_gla(C.byref(d), b.n, b.n_chunks, b.R, max(b.lens), _lib.ptr(b.seq_row0), _lib.ptr(b.seq_pos0), _lib.ptr(b.seq_slot),
                      _lib.ptr(b.seq_chunk0), _lib.ptr(b.chunk_seq), _lib.ptr(b.chunk_row0), _lib.ptr(b.chunk_len), _lib.ptr(ws), n_ws, eng._stream())
        eng._check(rc, "lp_gla")
        exp = torch.cat([want[k][at[k]:at[k] + n] for k, n in rows.items()], 0)
        assert float(_rows(out, exp).max()) < 10 * TOL["float32"], rows
        for s, n in zip(b.seqs, b.lens):
            eng.cache.advance(s, n)

    run({"a": lens[0], "b": lens[1]})
    run({"a": 2, "b": 3})
    run({"a": 1, "b": 1})
    # the low-rank form: one more token of "a" whose decay comes from t, w2 and the bias
    k = "a"
    n = eng.cache.get(k).length
    act = torch.tanh(data[k]["t"][n:n + 1].double()) if bonus else data[k]["t"][n:n + 1].double()
    z = (act @ w2.double().T + zb.double()).float()
    before = state.clone()
    outs = []
    for low_rank in (False, True):
        state.copy_(before)
        b = _Batch(eng, [StepEntry(k, [0])])
        row = {f: data[k][f][n:n + 1].to(dev) for f in "qkvgt"}
        zd, out = z.to(dev), torch.empty(1, H * vdim, device=dev)
        d = _lib.GlaDesc(q=_lib.ptr(row["q"]), k=_lib.ptr(row["k"]), v=_lib.ptr(row["v"]), ldq=H * dim, ldk=H * dim, ldv=H * vdim, heads=H, dim=dim,
                         vdim=vdim, q_scale=0.3, decay=_lib.GLA_DECAY_DOUBLE_EXP if bonus else _lib.GLA_DECAY_SIGMOID_POW, decay_exp=0.25,
                         z=None if low_rank else _lib.ptr(zd), ldz=H * dim, t=_lib.ptr(row["t"]), ldt=rank, w2=_lib.ptr(w2_d), ldw2=rank, rank=rank,
                         t_tanh=int(bonus), z_bias=_lib.ptr(zb_d), bonus=_lib.ptr(u_d) if bonus else None, out_gain=_lib.ptr(gain_d), gain_stride=vdim,
                         gate=_lib.ptr(row["g"]), ldg=H * vdim, eps=1e-5, state=_lib.ptr(state), slot_stride=state.stride(0), out=_lib.ptr(out),
                         ldo=H * vdim, out_fp32=1)
        n_ws = int(L.lp_gla_workspace_bytes(1, 1, 1, H, dim, vdim))
        ws = torch.empty(n_ws // 4 + 1, device=dev)
        eng._check(L.lp_gla(C.byref(d), 1, 1, 1, 1, _lib.ptr(b.seq_row0), _lib.ptr(b.seq_pos0), _lib.ptr(b.seq_slot), None, None, None, None,
                            _lib.ptr(ws), n_ws, eng._stream()), "lp_gla")
        outs.append((out.cpu(), state[eng.cache.get(k).slot].cpu()))
    assert rel_err(outs[1][0], outs[0][0]) < TOL["float32"] and rel_err(outs[1][1], outs[0][1]) < TOL["float32"]


@pytest.mark.parametrize("n, width", [(1, 12), (2, 10), (3, 16), (4, 12), (6, 11)])
def test_hyper_connections_kernel(backend, n, width):
    """closing, opening, both, the plain sum of the copies, and the token-shifted operands of one-token steps against torch; wide rows
    (beyond the registers) on the GPU"""
    from leopard_b200 import _lib
    eng = _bare_engine(backend)
    dev, L, st = eng.device, eng.L, eng._stream()
    for D in (width, 4096 + 1024 + width) if dev.type == "cuda" else (width,):
        g = torch.Generator().manual_seed(D)
        M = 3
        x0, y = torch.randn(M, n, D, generator=g), torch.randn(M, D, generator=g)
        mix, out_w, in_w = torch.randn(n, n, generator=g), torch.randn(n, generator=g), torch.randn(n, generator=g)
        gain, mu, prev = torch.rand(D, generator=g) + 0.5, torch.rand(4, D, generator=g), torch.randn(5, D, generator=g)
        dd = {k: v.to(dev) for k, v in dict(y=y, mix=mix, out_w=out_w, in_w=in_w, gain=gain, mu=mu).items()}
        pos, slot = torch.tensor([3, 0, 9], dtype=torch.int32).to(dev), torch.tensor([4, 1, 0], dtype=torch.int32).to(dev)
        for close, opens, mixes, dtype in ((True, None, False, torch.float32), (False, "in", False, torch.float32), (True, "in", False, torch.bfloat16),
                                           (True, "sum", False, torch.float32), (True, "in", True, torch.float32), (False, "in", True, torch.bfloat16)):
            xw = torch.einsum("st,msd->mtd", mix.double(), x0.double()) + out_w.double()[:, None] * y.double()[:, None] if close else x0.double()
            h = O.rms(torch.einsum("s,msd->md", in_w.double(), xw) if opens == "in" else xw.sum(1), 1e-4) * gain.double()
            x, state = x0.clone().to(dev), prev.clone().to(dev)
            out = torch.empty(4 if mixes else 1, M, D, dtype=dtype, device=dev)
            d = _lib.HyperDesc(x=_lib.ptr(x), ldx=n * D, n=n, D=D, eps=1e-4)
            if close:
                d.y, d.ldy, d.mix, d.out_w = _lib.ptr(dd["y"]), D, _lib.ptr(dd["mix"]), _lib.ptr(dd["out_w"])
            if opens:
                d.in_w, d.gain, d.h, d.ldh = _lib.ptr(dd["in_w"]) if opens == "in" else None, _lib.ptr(dd["gain"]), _lib.ptr(out), D
                d.h_fp32 = int(dtype == torch.float32)
            if mixes:
                d.mu, d.n_mix, d.mix_stride, d.row_pos, d.row_slot = _lib.ptr(dd["mu"]), 4, M * D, _lib.ptr(pos), _lib.ptr(slot)
                d.state, d.slot_stride = _lib.ptr(state), D
            eng._check(L.lp_hyper_f32(C.byref(d), M, st), "lp_hyper_f32")
            assert rel_err(x, xw) < TOL["float32"]
            if not opens:
                continue
            tol = TOL["float32"] if dtype == torch.float32 else 4e-3
            if mixes:
                before = torch.stack([prev[4], torch.zeros(D), prev[0]]).double()      # the second row starts its request
                for i in range(4):
                    assert rel_err(out[i].float(), h + (before - h) * mu[i].double()) < tol
                assert rel_err(state[[4, 1, 0]], h) < TOL["float32"] and torch.equal(state[[2, 3]].cpu(), prev[[2, 3]])
            else:
                assert rel_err(out[0].float(), h) < tol


@pytest.mark.parametrize("experts, top, groups, keep", [(8, 3, 4, 2), (6, 1, 1, 1), (40, 5, 8, 3), (70, 4, 35, 33), (5, 5, 5, 5)])
def test_group_softmax_router(backend, experts, top, groups, keep):
    """chosen experts and weights of every token against the plain choice, both operand precisions"""
    from leopard_b200 import _lib
    eng = _bare_engine(backend)
    dev, T, D = eng.device, 9, 16
    g = torch.Generator().manual_seed(experts)
    h = torch.randn(T, D, generator=g).to(torch.bfloat16)
    wr = torch.randn(experts, D, generator=g).to(torch.bfloat16)
    want = O.route(h.double(), {"router": wr.double()}, "", {"experts": experts, "top": top, "scale": 1.7, "groups": {"count": groups, "keep": keep}})
    wr = wr.to(dev)
    for hh in (h.to(dev), h.float().to(dev)):
        idx, wt = torch.empty(T, top, dtype=torch.int32, device=dev), torch.empty(T, top, device=dev)
        rc = eng.L.lp_moe_route_group_softmax(_lib.ptr(hh), D, int(hh.dtype == torch.float32), T, D, _lib.ptr(wr), D, experts, groups, keep, top, 1.7,
                                              _lib.ptr(idx), _lib.ptr(wt), eng._stream())
        eng._check(rc, "lp_moe_route_group_softmax")
        for t in range(T):
            got = dict(zip(idx[t].tolist(), wt[t].tolist()))
            assert set(got) == set(want[t])
            assert all(math.isclose(got[e], want[t][e], rel_tol=1e-5) for e in got)
    assert eng.L.lp_moe_route_group_softmax(_lib.ptr(hh), D, 1, T, D, _lib.ptr(wr), D, experts, experts + 1, 1, top, 1.0, _lib.ptr(idx), _lib.ptr(wt),
                                            eng._stream()) != 0


@pytest.mark.parametrize("rows", [3, 70])
@pytest.mark.parametrize("seg", [8, 64, 5])
def test_column_segments_of_a_product(backend, rows, seg):
    """columns that read operands of their own, in one launch where the segments fit its CTAs and one by one elsewhere"""
    eng = _bare_engine(backend)
    g = torch.Generator().manual_seed(seg)
    ops = torch.randn(3, rows, 12, generator=g)
    w = torch.randn(2 * seg + 11, 12, generator=g).to(torch.bfloat16)
    got = eng.linear_segments(ops.to(eng.device), w.to(eng.device), seg)
    want = torch.cat([ops[i].double() @ w[a:b].double().T for i, (a, b) in enumerate([(0, seg), (seg, 2 * seg), (2 * seg, 2 * seg + 11)])], 1)
    assert rel_err(got, want) < TOL["float32"]


@pytest.mark.parametrize("split", [0, 1])
def test_low_rank_operand(backend, split):
    from leopard_b200 import _lib
    eng = _bare_engine(backend)
    t = torch.randn(5, 9, generator=torch.Generator().manual_seed(1))
    td = t.to(eng.device)
    out = torch.zeros(5, 16, dtype=torch.bfloat16 if split else torch.float32, device=eng.device)
    rc = eng.L.lp_lowrank_operand(_lib.ptr(td), 9, 5, 7, 1, _lib.ptr(out), 16, split, eng._stream())
    eng._check(rc, "lp_lowrank_operand")
    got = out[:, :7].double().cpu() + (out[:, 7:14].double().cpu() if split else 0)
    assert float((got - torch.tanh(t[:, :7].double())).abs().max()) < (2e-5 if split else 1e-6)


def test_the_attention_options_in_other_combinations(backend):
    """the options of the windowed attention one by one beside others: a convolution with values of their own, a gate on the plain
    kernels with a sink and kept first tokens, slopes without a gate over everything, a position temperature beside a head norm"""
    from leopard_b200.seqlm import LayerConfig, RotaryConfig, SeqLMConfig, SeqLMEngine, SeqLMWeights, WindowAttentionConfig
    device, lib = backend
    none = RotaryConfig(dims=0, base=1.0)
    H, G, d, e, D = 4, 2, 6, 5, 10
    for kw in (dict(qk_conv=3, window=4, out_gate=True), dict(out_gate=True, sink=True, window=3, keep_first=2), dict(distance_slope=True),
               dict(distance_slope=True, window=4, keep_first=1, out_gate=True), dict(pos_temp=(0.5, 2), qk_norm="head", window=5)):
        m = WindowAttentionConfig(heads=H, kv_heads=G, dim=d, vdim=e, scale=0.7, rot=none, **kw)
        cfg = SeqLMConfig("test", 23, D, 1e-5, (LayerConfig(m, None),), norm="pre_plain", learned_positions=20)
        g = torch.Generator().manual_seed(5)
        w = {n: (torch.randn(*s, generator=g) / math.sqrt(s[-1]) * 1.5).to(torch.bfloat16).float() for n, s in {
            "embed": (23, D), "pos": (20, D), "head": (23, D), "l0.mix.q": (H * d, D), "l0.mix.k": (G * d, D), "l0.mix.v": (G * e, D),
            "l0.mix.g": (H * e, D), "l0.mix.o": (D, H * e), "l0.mix.q.conv": (H * d, 3), "l0.mix.k.conv": (G * d, 3)}.items()}
        for n, s in (("final.norm", D), ("l0.norm1", D), ("l0.mix.q.norm", d), ("l0.mix.k.norm", d)):
            w[n] = (1 + 0.3 * torch.randn(s, generator=g)).to(torch.bfloat16).float()
        T = 12
        toks = _tokens(T, 23, seed=9)
        f = {k: v.double() for k, v in w.items()}
        x = f["embed"][torch.tensor(toks)] + f["pos"][:T]
        h = O.rms(x, 1e-5) * f["l0.norm1"]
        q, k, v = h @ f["l0.mix.q"].T, h @ f["l0.mix.k"].T, (h @ f["l0.mix.v"].T).view(T, G, e)
        if m.qk_conv:
            q, k = O.causal_conv(q, f["l0.mix.q.conv"]), O.causal_conv(k, f["l0.mix.k.conv"])
        q, k = q.view(T, H, d), k.view(T, G, d)
        if m.qk_norm == "head":
            q, k = O.rms(q, 1e-5) * f["l0.mix.q.norm"], O.rms(k, 1e-5) * f["l0.mix.k.norm"]
        y = torch.zeros(T, H, e, dtype=torch.float64)
        for i in range(T):
            for hd in range(H):
                see = [j for j in range(i + 1) if m.window is None or i - j < m.window or j < m.keep_first]
                temp = 1 + m.pos_temp[0] * math.log((i + 1) // m.pos_temp[1] + 1) if m.pos_temp else 1.0
                s = torch.stack([temp * (q[i, hd] @ k[j, hd // 2]) * 0.7 - (2.0 ** (-8 * (hd + 1) / H) * (i - j) if m.distance_slope else 0.0) for j in see])
                p = torch.softmax(torch.cat([s, torch.zeros(1, dtype=torch.float64)]) if m.sink else s, 0)
                y[i, hd] = sum(p[a] * v[j, hd // 2] for a, j in enumerate(see))
        y = y.reshape(T, H * e)
        if m.out_gate:
            y = y * torch.sigmoid(h @ f["l0.mix.g"].T)
        want = (O.rms(x + y @ f["l0.mix.o"].T, 1e-5) * f["final.norm"]) @ f["head"].T
        eng = SeqLMEngine(cfg, SeqLMWeights(cfg, lambda n: w[n], bezizen.tensor_name, device), dtype="float32", max_tokens=32, page_size=4,
                          max_seqs=2, lib=lib)
        assert float(_rows(_prompt_then_decode(eng, toks, 7), want).max()) < 5 * TOL["float32"], kw


def test_memories_in_other_layer_forms(backend):
    """the time mixing and the gated linear attention as plain mixers of a pre-norm stack with one stream"""
    from leopard_b200.seqlm import GatedLinearConfig, LayerConfig, SeqLMConfig, SeqLMEngine, SeqLMWeights, WKVConfig
    base = model([wkv_layer(), parallel_layer()])
    w = O.random_weights(base, seed=51)
    device, lib = backend
    cfg = SeqLMConfig("test", 41, 12, 1e-5, (LayerConfig(WKVConfig(heads=2, dim=6), None), LayerConfig(GatedLinearConfig(heads=3, dim=6, vdim=5, tau=4.0), None)),
                      norm="pre_plain", residual_mult=0.6)
    toks = _tokens(9, 41, seed=53)
    d = {k: v.double() for k, v in w.items()}
    x = d["embed"][torch.tensor(toks)]
    x = x + 0.6 * O.wkv_mixer(O.rms(x, 1e-5) * d["l0.norm1"], d, "l0.mix.", base["layers"][0]["mixer"], 1e-5)
    x = x + 0.6 * O.gated_linear_attention(O.rms(x, 1e-5) * d["l1.norm1"], d, "l1.mix.right.", base["layers"][1]["mixer"]["right"], 1e-5)
    want = (O.rms(x, 1e-5) * d["final.norm"]) @ d["head"].T
    eng = SeqLMEngine(cfg, SeqLMWeights(cfg, lambda n: w[n.replace("l1.mix.", "l1.mix.right.")], bezizen.tensor_name, device), dtype="float32",
                      max_tokens=32, page_size=4, max_seqs=2, lib=lib)
    assert float(_rows(_prompt_then_decode(eng, toks, 4), want).max()) < 5 * TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_are_equal_or_one(backend, dtype):
    """one head everywhere, one stream, a window of one token, one tap, rank one, one expert that is always chosen, scales of one, a query
    temperature without effect, an odd width"""
    layers = [wkv_layer(heads=1, dim=9, rank=1, mlp=moe(experts=1, top=1, groups=(1, 1), ff=1, shared=1, scale=1.0)),
              parallel_layer(heads=1, kv_heads=1, dim=9, conv=1, window=1, scale=1.0, coef=0.0, every=1, left=1.0, right=1.0, gheads=1, gdim=1, gvdim=1,
                             tau=1.0, rank=1)]
    cfg = model(layers, width=9, vocab=23, eps=1e-6, embed=1.0, streams=1, positions=6, logit_scale=1.0)
    w = O.random_weights(cfg, seed=24)
    toks = _tokens(6, 23, seed=10)
    want = O.forward(cfg, w, toks)
    eng = make_engine(cfg, w, backend, dtype)
    assert rel_err(_prompt_then_decode(eng, toks, 3), want) < TOL[dtype]
    with pytest.raises(ValueError, match="positions"):           # the table of learned positions ends here
        eng.step([StepEntry("r", [0], [0])])
    with pytest.raises(ValueError, match="positions"):
        eng.step([StepEntry("s", [0] * 7, [])])
    assert eng.cache.get("s") is None


def test_greedy_generation_through_the_scheduler(backend):
    cfg = mixed_model()
    w = O.random_weights(cfg, seed=19)
    prompts = [_tokens(n, cfg["vocab"], seed=40 + n) for n in (3, 5, 1)]
    eng = make_engine(cfg, w, backend, max_seqs=2)
    outs = generate(eng, prompts, max_new_tokens=3)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for t in o:                                   # every generated token is the oracle's arg-max given what came before
            lg = O.forward(cfg, w, seq)[-1]
            top2 = lg.topk(2).values
            assert int(lg.argmax()) == t or float(top2[0] - top2[1]) < 1e-3
            seq.append(t)
        assert len(o) == 3
    assert eng.cache.pages_in_use() == 0
    sched = Scheduler(eng, max_running=1)
    first = outs[0][0]
    sched.add(Request("x", prompts[0], max_new_tokens=2, eos={first}))
    sched.add(Request("y", prompts[1], max_new_tokens=1))
    done = sched.run()
    assert done["x"].output == [first] and done["y"].output == outs[1][:1]


@pytest.mark.gpu
def test_command_line_generate_and_trace(tmp_path):
    """the registry picks the loader from config.json; `generate` and `trace` run the same step engine"""
    import subprocess
    import sys
    from pathlib import Path
    import numpy as np
    from leopard_b200.safetensors_io import save_file
    root = Path(__file__).resolve().parents[1]
    cfg = mixed_model()
    w = O.random_weights(cfg, seed=20)
    (tmp_path / "m").mkdir()
    (tmp_path / "m/config.json").write_text(json.dumps(cfg))
    save_file(w, tmp_path / "m/model.safetensors")
    toks = _tokens(12, cfg["vocab"], seed=8)
    r = subprocess.run([sys.executable, "-m", "leopard_b200", "generate", "--model", str(tmp_path / "m"), "--dtype", "float32", "--prompt",
                        ",".join(map(str, toks)), "--max-new-tokens", "3"], cwd=root, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr[-2000:]
    out = json.loads(r.stdout.strip().splitlines()[-1])["output"]
    assert out[0] == int(O.forward(cfg, w, toks)[-1].argmax())
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": toks[:9], "want": [0, 8]}, {"id": "s", "tokens": toks[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": toks[9:10], "want": []}, {"id": "s", "tokens": toks[2:3], "want": [0]}],
              "end": ["s"]},
             {"step": 2, "entries": [{"id": "q", "tokens": toks[10:11], "want": [0]}], "end": ["q"]}]
    for dtype in ("float32", "bfloat16"):
        r = subprocess.run([str(root / "bin/trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path / dtype),
                            "--max-tokens", "64"], input="\n".join(map(json.dumps, steps)) + "\n", cwd=root, capture_output=True, text=True)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        want = O.forward(cfg, w, toks)
        got = [torch.from_numpy(np.fromfile(tmp_path / dtype / f"{i}.f32", dtype="<f4").reshape(n, -1)) for i, n in ((0, 2), (1, 1), (2, 1))]
        assert rel_err(got[0], want[[0, 8]]) < TOL[dtype] and rel_err(got[1], want[2:3]) < TOL[dtype]
        assert rel_err(got[2], want[10:11]) < TOL[dtype]


def test_registry_and_config_reader():
    from leopard_b200 import registry
    from leopard_b200.seqlm import GatedLinearConfig, MoEConfig, ParallelMixerConfig, WindowAttentionConfig, WKVConfig
    assert "Bezizen" in registry.architectures()
    cfg = bezizen.config_from_dict(mixed_model())
    assert (cfg.norm, cfg.streams, cfg.learned_positions, cfg.logit_scale, cfg.embed_scale, cfg.eps) == ("pre_plain", 3, 300, 0.6, 1.5, 1e-5)
    a, b, c = cfg.layers
    assert isinstance(a.mixer, WKVConfig) and (a.mixer.heads, a.mixer.dim) == (2, 6) and c.ff is None
    assert isinstance(a.ff, MoEConfig) and (a.ff.router, a.ff.experts, a.ff.top, a.ff.n_groups, a.ff.keep_groups, a.ff.weight_scale, a.ff.expert_ff,
                                            a.ff.shared_ff, a.ff.shared_gate) == ("group_softmax", 6, 3, 3, 2, 1.6, 5, 7, False)
    assert (b.ff.n_groups, b.ff.keep_groups, b.ff.shared_ff, b.ff.weight_scale) == (1, 1, 0, 0.8)
    m = b.mixer
    assert isinstance(m, ParallelMixerConfig) and isinstance(m.left, WindowAttentionConfig) and isinstance(m.right, GatedLinearConfig)
    assert m.scales == (1.2, 0.7) and (m.left.heads, m.left.kv_heads, m.left.dim, m.left.vdim, m.left.window, m.left.qk_conv, m.left.pos_temp) == \
        (4, 2, 8, 8, 5, 3, (0.4, 3))
    assert m.left.values_are_keys and m.left.distance_slope and m.left.out_gate and m.left.rot.dims == 0 and m.left.scale == 0.5
    assert (m.right.heads, m.right.dim, m.right.vdim, m.right.tau) == (3, 6, 5, 4.0)
    assert bezizen.tensor_name(3, "hc2.mix") == "l3.hc2.mix" and bezizen.tensor_name(None, "pos") == "pos"
    with pytest.raises(ValueError):
        bezizen.config_from_dict({"architecture": "other"})
    bad = mixed_model()
    bad["layers"][1]["mixer"]["left"]["vdim"] = 7
    with pytest.raises(ValueError, match="vdim"):
        bezizen.config_from_dict(bad)


def test_shapes_are_checked(emu_lib):
    """a tensor that does not fit the configuration is named"""
    cfg = mixed_model()
    for name in ("l0.hc1.mix", "l0.mix.w2", "l1.mix.left.k.conv", "l1.mix.right.a2", "pos"):
        w = O.random_weights(cfg, seed=1)
        w[name] = w[name][:-1]
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            make_engine(cfg, w, ("cpu", emu_lib))
