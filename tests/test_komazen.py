"""Komazen on the step engine against the plain implementation (oracle/komazen.py): every mechanism alone, whole prompts against
token-by-token decoding, prompts cut into portions down to one and two tokens (fewer than the convolution looks back), batches of unequal
requests, pages and slots that are given back and taken again, keys just inside and just outside a window (in a prompt and decoded, in
a layer with latents of its own and in one that reads another layer's), page borders, far keys under the distance bias, the first
tokens of a sequence, long decoding, sizes that happen to be equal or one, both precisions, and greedy generation through the
scheduler and the command line.  Where random weights would hide a fault, the configuration's score scale is raised so that every
softmax leans on few keys, or one key is made to stand out, and the test first shows on the oracle itself that the fault would be
noticed.  On the kernel sources under the CPU emulator and, marked gpu, on the native library."""
import copy
import json

import pytest
import torch

from leopard_b200 import komazen
from leopard_b200.scheduler import Request, Scheduler, generate
from leopard_b200.seqlm import StepEntry
from oracle import komazen as O
from komazen_common import TOL, attention_layer, backend, dense, emu_lib, latent_layer, make_engine, mixed_model, model, rel_err  # noqa: F401


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
    "latent": ([latent_layer()], {}),
    "latent, odd sizes, one head, long convolution": ([latent_layer(heads=1, dim=3, rot_dim=2, vdim=7, q_rank=5, kv_rank=33, window=3)],
                                                     {"taps": 6, "width": 11}),
    "latent + dense": ([latent_layer(mlp=dense())], {}),
    "two latent layers on one set of latents": ([latent_layer(), latent_layer(heads=3, dim=4, vdim=3, window=7, kv_from=0)], {}),
    "attention": ([attention_layer()], {}),
    "attention, odd sizes, one key head": ([attention_layer(heads=3, kv_heads=1, dim=6, vdim=7)], {"taps": 2}),
    "attention, every head its own keys, one tap": ([attention_layer(heads=2, kv_heads=2, dim=16, vdim=16)], {"taps": 1}),
    "attention + dense": ([attention_layer(mlp=dense(ff=9))], {"taps": 4, "width": 16}),
}


@pytest.mark.parametrize("name", list(MODELS))
def test_each_mechanism_alone(backend, name):
    """a small model: the whole prompt in one step, and the same tokens with the last ones decoded through cache and state"""
    layers, kw = MODELS[name]
    cfg = model(layers, **kw)
    w = O.random_weights(cfg, seed=3)
    toks = _tokens(8, cfg["vocab"], seed=1)
    res = []
    want = O.forward(cfg, w, toks, taps=res)
    eng = make_engine(cfg, w, backend)
    taps = []
    eng.tap = lambda li, x: taps.append(x.clone())
    got = eng.step([StepEntry("p", toks, _all(8))])
    assert len(taps) == len(res)
    for a, b in zip(taps, res):                                   # the stream after every layer
        assert rel_err(a, b) < TOL["float32"]
    assert float(_rows(got, want).max()) < 5 * TOL["float32"]
    eng.tap = None
    eng.finish("p")
    assert float(_rows(_prompt_then_decode(eng, toks, 5), want).max()) < 5 * TOL["float32"]


def test_every_piece_matters_on_the_oracle():
    """each piece, shown to move the logits when it is left out or changed"""
    cfg = mixed_model()
    w = O.random_weights(cfg, seed=4)
    toks = _tokens(9, cfg["vocab"], seed=5)
    want = O.forward(cfg, w, toks)
    changes = {"l0.canon1": 0.0, "l0.canon2": 0.0, "l1.canon1": 0.0, "l2.canon1": 0.0, "l0.norm1": 1.0, "l2.norm2": 1.0, "final.norm": 1.0,
               "l0.mix.g": 0.0, "l2.mix.g": 0.0, "l0.mix.dq.norm": 1.0, "l0.mix.dkv.norm": 1.0, "l1.mix.temp": 1.0, "l1.mix.r1": 0.0,
               "l1.mix.r2": 0.05, "l1.mix.q.norm": 1.0, "l1.mix.k.norm": 1.0, "l0.mlp.gate": 0.0}
    for name, value in changes.items():
        w2 = dict(w)
        w2[name] = torch.full_like(w[name], value)
        assert float(_rows(O.forward(cfg, w2, toks), want).median()) > 200 * TOL["float32"], name
    for path, value in ((("postln_alpha",), 1.7), (("embedding", "scale"), 1.4), (("norm", "eps"), 1e-2),
                        (("layers", 0, "mixer", "scale"), 0.45), (("layers", 1, "mixer", "scale"), 0.55),
                        (("layers", 2, "mixer", "rot", "base"), 50.0)):
        c2 = copy.deepcopy(cfg)
        node = c2
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        assert float(_rows(O.forward(c2, w, toks), want).median()) > 20 * TOL["float32"], path


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_then_long_decoding(backend, dtype):
    """a prompt, then tokens one by one: windows pass over decoded tokens, pages fill up, the convolutions' inputs are carried"""
    cfg = mixed_model(taps=4)
    w = O.random_weights(cfg, seed=11)
    toks = _tokens(90, cfg["vocab"], seed=2)
    want = O.forward(cfg, w, toks)
    eng = make_engine(cfg, w, backend, dtype, max_tokens=96)
    got = _prompt_then_decode(eng, toks, 21)
    assert rel_err(got, want) < TOL[dtype]
    if dtype == "float32":
        assert float(_rows(got, want).max()) < 5 * TOL[dtype]


@pytest.mark.parametrize("cuts", [(2, 2, 3, 2), (1, 2, 8), (5, 36, 2, 33, 3)])
def test_portions_of_a_prompt(backend, cuts):
    """a prompt fed in portions, some shorter than the convolution looks back (5 taps), some longer than a 32-row chunk"""
    cfg = mixed_model(taps=5)
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
    pages and the slot that were given back (the pools are sized so that it must), whose carried inputs it must not see"""
    cfg = mixed_model()
    w = O.random_weights(cfg, seed=13)
    lens = {"a": (1, 2), "b": (5, 3), "c": (7, 1)}            # prompt length, decoded tokens
    toks = {k: _tokens(p + d, cfg["vocab"], seed=30 + i) for i, (k, (p, d)) in enumerate(lens.items())}
    want = {k: O.forward(cfg, w, toks[k]) for k in lens}
    eng = make_engine(cfg, w, backend, max_tokens=8, max_seqs=3)
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


def _one_off(cfg, delta, layer=None):
    c = copy.deepcopy(cfg)
    for i, l in enumerate(c["layers"]):
        if "mask" in l["mixer"] and layer in (None, i):
            l["mixer"]["mask"]["size"] += delta
    return c


@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("mode", ["prompt", "decoded"])
def test_edge_of_the_window(backend, shared, mode):
    """a large score scale makes every softmax lean on few keys: the oracle with a window one token longer or shorter differs by far
    more than the tolerance on many rows, and the engine agrees with the right one — in a layer with latents of its own and in one
    that reads another layer's, whose window is longer than the owner's, across page borders (pages of 4 tokens), with the pages
    behind the longest window given back while the request runs"""
    layers = [latent_layer(window=4, scale=3.0)]
    if shared:
        layers.append(latent_layer(window=6, scale=3.0, kv_from=0))
    cfg = model(layers)
    w = O.random_weights(cfg, seed=21)
    toks = _tokens(41, cfg["vocab"], seed=6)
    want = O.forward(cfg, w, toks)
    for delta in (-1, 1):
        off = _rows(O.forward(_one_off(cfg, delta, len(layers) - 1), w, toks), want)
        edge = layers[-1]["mixer"]["mask"]["size"] + min(delta, 0)
        assert int((off[edge:] > 200 * TOL["float32"]).sum()) >= 8
        assert float(off[:edge].max()) < 1e-12                      # rows that see the same either way
    eng = make_engine(cfg, w, backend, max_tokens=8)
    got = eng.step([StepEntry("r", toks, _all(41))]) if mode == "prompt" else _prompt_then_decode(eng, toks, 3)
    assert float(_rows(got, want).max()) < 5 * TOL["float32"]
    assert sum(p >= 0 for p in eng.cache.get("r").pages) <= 3      # only the pages of the longest window are still held


def test_attention_over_everything_keeps_every_page(backend):
    """one causal layer among windowed ones: no page is given back, and the first token still counts at the end"""
    cfg = model([latent_layer(window=2), attention_layer(scale=2.0)])
    w = O.random_weights(cfg, seed=25)
    w["l1.mix.r1"] = torch.full_like(w["l1.mix.r1"], 0.05)      # hardly any bias: far keys carry weight
    toks = _tokens(14, cfg["vocab"], seed=26)
    want = O.forward(cfg, w, toks)
    other = O.forward(cfg, w, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    assert float(_rows(other[-3:], want[-3:]).max()) > 100 * TOL["float32"]
    eng = make_engine(cfg, w, backend, max_tokens=8)
    assert float(_rows(_prompt_then_decode(eng, toks, 10), want).max()) < 5 * TOL["float32"]
    assert all(p >= 0 for p in eng.cache.get("r").pages)


@pytest.mark.gpu
def test_far_keys_and_edges_among_hundreds():
    """windows of hundreds of keys and causal attention over everything (several key tiles, many pages), sharp softmaxes: the oracle
    with a window one token off and a changed first token is told apart; portions start at every kind of
    offset and the end is decoded"""
    layers = [latent_layer(heads=16, dim=8, rot_dim=8, vdim=8, q_rank=12, kv_rank=16, window=150, scale=0.7),
              attention_layer(heads=8, kv_heads=2, dim=16, vdim=8, scale=1.0),
              latent_layer(heads=12, dim=8, rot_dim=8, vdim=8, q_rank=12, kv_rank=16, window=131, scale=0.7, kv_from=0)]
    cfg = model(layers, width=24, taps=4, alpha=1.5)
    w = O.random_weights(cfg, seed=31)
    w["l1.mix.r1"] = w["l1.mix.r1"] * 0.2
    toks = _tokens(330, cfg["vocab"], seed=32)
    want = O.forward(cfg, w, toks)
    for li in (0, 2):
        for delta in (-1, 1):
            off = _rows(O.forward(_one_off(cfg, delta, li), w, toks), want)
            assert int((off[150:] > 200 * TOL["float32"]).sum()) >= 15
    first = O.forward(cfg, w, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])      # the causal layer remembers token 0
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
    assert rel_err(both[1:], want[:300]) < TOL["bfloat16"]
    alone = half.step([StepEntry("z", toks[:300], _all(300))])
    assert rel_err(both[1:], alone) < 5e-3


@pytest.mark.parametrize("taps", [2, 4, 8, 11])
def test_convolution_carries_its_inputs(backend, taps):
    """the causal convolution kernel alone against the oracle: a request cut into every kind of portion, a second request beside it,
    stale slots, widths of the four-channel and the one-channel path, taps inside and beyond the register window; then the one-token
    form that rides on the post-norm"""
    from leopard_b200 import _lib
    from leopard_b200.seqlm import _Batch
    for width in (12, 10):
        cfg = model([attention_layer(heads=1, kv_heads=1, dim=4, vdim=4)], width=width, taps=taps)
        w = O.random_weights(cfg, seed=taps)
        eng = make_engine(cfg, w, backend, max_tokens=128)
        for st in eng.cache.states:
            st.fill_(7.0)                                         # what an earlier request may have left
        g = torch.Generator().manual_seed(taps)
        n = 44
        h = {k: O.rms_norm(torch.randn(n, width, generator=g), 1.0, 0.0) for k in "ab"}
        want = {k: O.with_convolution(h[k].double(), w["l0.canon1"].double()) for k in "ab"}
        at = {"a": 0, "b": 0}
        for na, nb in ((1, 2), (2, 1), (3, 4), (33, 5), (1, 1), (2, 1)):
            entries = [StepEntry(k, [0] * m) for k, m in (("a", na), ("b", nb))]
            b = _Batch(eng, entries)
            rows = torch.cat([h[k][at[k]:at[k] + m] for k, m in (("a", na), ("b", nb))], 0).to(eng.device)
            exp = torch.cat([want[k][at[k]:at[k] + m] for k, m in (("a", na), ("b", nb))], 0)
            if b.decode:      # alpha 0 and unit gain: the rows, of root mean square one, pass the norm as they are
                x, out, gain = torch.zeros_like(rows), torch.empty_like(rows), torch.ones(width, device=eng.device)
                st = eng._conv_state(0, "conv1")
                rc = eng.L.lp_post_norm_f32(_lib.ptr(x), width, _lib.ptr(rows), width, 0.0, 2, width, _lib.ptr(gain), 0.0, _lib.ptr(out), width, 1,
                                            _lib.ptr(eng.w.layers[0]["conv1"]), taps, _lib.ptr(b.row_pos), _lib.ptr(b.seq_slot), _lib.ptr(st),
                                            st.stride(0), eng._stream())
                eng._check(rc, "lp_post_norm_f32")
                assert rel_err(out, exp) < TOL["float32"] and rel_err(x, rows) < TOL["float32"]
            else:
                got = eng.convolved(rows, 0, "conv1", b)
                assert rel_err(got, exp) < TOL["float32"]
            for s, m in zip(b.seqs, b.lens):
                eng.cache.advance(s, m)
            at["a"] += na
            at["b"] += nb


@pytest.mark.parametrize("width", [12, 10])
def test_post_norm_kernel(backend, width):
    """norm after the sum against torch: with and without the operand, both operand precisions, wide rows (beyond the registers) on
    the GPU"""
    from leopard_b200 import _lib
    cfg = model([attention_layer(heads=1, kv_heads=1, dim=4, vdim=4)])
    eng = make_engine(cfg, O.random_weights(cfg, seed=1), backend)
    dev, L, st = eng.device, eng.L, eng._stream()
    for D in (width, 4096 + 1024 + width) if dev.type == "cuda" else (width,):
        g = torch.Generator().manual_seed(D)
        x0, y = torch.randn(3, D, generator=g), torch.randn(3, D, generator=g)
        gain = torch.rand(D, generator=g) + 0.5
        want = O.rms_norm(1.3 * x0.double() + y.double(), gain.double(), 1e-4)
        y, gain = y.to(dev), gain.to(dev)
        for dtype in (None, torch.float32, torch.bfloat16):
            x = x0.clone().to(dev)
            out = torch.empty(3, D, dtype=dtype, device=dev) if dtype is not None else None
            rc = L.lp_post_norm_f32(_lib.ptr(x), D, _lib.ptr(y), D, 1.3, 3, D, _lib.ptr(gain), 1e-4, _lib.ptr(out), D,
                                    int(dtype == torch.float32), None, 0, None, None, None, 0, st)
            eng._check(rc, "lp_post_norm_f32")
            if dev.type == "cuda":
                torch.cuda.synchronize()
            assert rel_err(x, want) < TOL["float32"]
            if out is not None:
                assert rel_err(out.float(), want) < (TOL["float32"] if dtype == torch.float32 else 4e-3)


@pytest.mark.parametrize("rows", [3, 70])
def test_gelu_unit_and_gated_heads(backend, rows):
    """the gelu-gated epilogue of the product (weight-streaming kernel and tile kernel), the same unit after a product, and per-head
    products whose result passes a gate"""
    from leopard_b200 import _lib
    cfg = model([attention_layer(heads=1, kv_heads=1, dim=4, vdim=4)])
    eng = make_engine(cfg, O.random_weights(cfg, seed=1), backend)
    dev = eng.device
    g = torch.Generator().manual_seed(rows)
    K, N = 12, 14
    a = 3 * torch.randn(rows, K, generator=g)
    w = torch.randn(N, K, generator=g).to(torch.bfloat16)
    z = a.double() @ w.double().T
    want = O.gelu_tanh(z[:, : N // 2]) * z[:, N // 2:]
    assert float(z[:, : N // 2].min()) < -12 and float(z[:, : N // 2].max()) > 12      # both ends of the unit
    assert rel_err(eng.linear(a.to(dev), w.to(dev), torch.float32, _lib.EPI_GELU_GATE), want) < TOL["float32"]
    zf, out = z.float().to(dev), torch.empty(rows, N // 2, device=dev)
    rc = eng.L.lp_glu_f32(_lib.ptr(zf), N, 1, _lib.ptr(out), N // 2, 1, rows, N // 2, _lib.EPI_GELU_GATE, 0.0, 0.0, eng._stream())
    eng._check(rc, "lp_glu_f32")
    assert rel_err(out, want) < TOL["float32"]
    wh = torch.randn(3, 5, 4, generator=g).to(torch.bfloat16)      # three heads, 4 -> 5
    wide = torch.randn(rows, 20, generator=g)
    gate = wide[:, 3:18]
    o = torch.empty(rows, 15, device=dev)
    eng.linear_heads(a.to(dev), 4, wh.to(dev), o, 5, gate=wide.to(dev)[:, 3:18])
    want = torch.cat([a[:, 4 * i:4 * i + 4].double() @ wh[i].double().T for i in range(3)], 1) * torch.sigmoid(gate.double())
    assert rel_err(o, want) < TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_are_equal_or_one(backend, dtype):
    """one head everywhere, a window of one token, latents as wide as the model, an alpha, an embedding scale and a temperature of
    one, a distance rate and amplitude of zero, a width that is odd, one tap"""
    layers = [latent_layer(heads=1, dim=4, rot_dim=4, vdim=4, q_rank=9, kv_rank=9, window=1, mlp=dense(ff=9)),
              latent_layer(heads=1, dim=4, rot_dim=4, vdim=4, q_rank=4, kv_rank=9, window=2, kv_from=0),
              attention_layer(heads=1, kv_heads=1, dim=4, vdim=4, scale=1.0, mlp=dense(ff=1))]
    cfg = model(layers, width=9, vocab=23, eps=1e-6, alpha=1.0, embed=1.0, taps=1)
    w = O.random_weights(cfg, seed=24)
    w["l2.mix.temp"], w["l2.mix.r1"], w["l2.mix.r2"] = torch.ones(1), torch.zeros(1), torch.zeros(1)
    toks = _tokens(6, 23, seed=10)
    want = O.forward(cfg, w, toks)
    eng = make_engine(cfg, w, backend, dtype)
    assert not eng.cache.states                                   # one tap carries nothing
    assert rel_err(_prompt_then_decode(eng, toks, 3), want) < TOL[dtype]


@pytest.mark.gpu
def test_wide_layers_on_the_tensor_cores():
    """sizes at which the serving precision sends its products to the tcgen05 GEMM, with the unit after the product and the operand of
    the next sublayer in 16 bits"""
    layers = [latent_layer(heads=4, dim=32, rot_dim=16, vdim=32, q_rank=64, kv_rank=128, window=100, scale=0.15, mlp=dense(ff=256)),
              attention_layer(heads=8, kv_heads=2, dim=32, vdim=48, scale=0.2, mlp=dense(ff=256)),
              latent_layer(heads=4, dim=32, rot_dim=16, vdim=32, q_rank=128, kv_rank=128, window=90, scale=0.15, kv_from=0)]
    cfg = model(layers, width=128, vocab=300, taps=4)
    w = O.random_weights(cfg, seed=41)
    toks = _tokens(300, cfg["vocab"], seed=42)
    want = O.forward(cfg, w, toks)
    for dtype in ("float32", "bfloat16"):
        eng = make_engine(cfg, w, ("cuda", None), dtype, max_tokens=512, page_size=64)
        got = eng.step([StepEntry("r", toks[:280], _all(280))])
        assert rel_err(got, want[:280]) < TOL[dtype], dtype
        more = torch.cat([eng.step([StepEntry("r", [t], [0])]) for t in toks[280:]], 0)
        assert rel_err(more, want[280:]) < TOL[dtype], dtype


@pytest.mark.parametrize("shift", [False, True])
def test_convolutions_in_other_layer_forms(backend, shift):
    """the input convolution under a norm ahead of the sublayer, alone and after the token shift: a pre-norm stack of the same
    attention, prompt and decoding"""
    from leopard_b200.seqlm import DenseFFConfig, LayerConfig, SeqLMConfig, SeqLMEngine, SeqLMWeights
    base = model([attention_layer(mlp=dense())], taps=3)
    w = O.random_weights(base, seed=51)
    g = torch.Generator().manual_seed(52)
    w["l0.shift"] = torch.rand(12, generator=g)
    kz = komazen.config_from_dict(base)
    cfg = SeqLMConfig(architecture="test", vocab=41, width=12, eps=1e-5, norm="pre", residual_mult=0.6, embed_scale=1.5,
                      layers=(LayerConfig(mixer=kz.layers[0].mixer, ff=DenseFFConfig(ff=10, act="gelu_glu"), input_conv=3, token_shift=shift),))
    toks = _tokens(7, 41, seed=53)
    d = {k: v.double() for k, v in w.items()}
    x = d["embed"][torch.tensor(toks)] * 1.5
    h = O.rms_norm(x, 1.0 + d["l0.norm1"], 1e-5)
    if shift:
        h = h + (torch.cat([torch.zeros(1, 12), h[:-1]]) - h) * d["l0.shift"]
    x = x + 0.6 * O.biased_attention(O.with_convolution(h, d["l0.canon1"]), d, "l0.mix.", base["layers"][0]["mixer"], 1e-5)
    x = x + 0.6 * O.feed_forward(O.with_convolution(O.rms_norm(x, 1.0 + d["l0.norm2"], 1e-5), d["l0.canon2"]), d, "l0.mlp.")
    want = O.rms_norm(x, 1.0 + d["final.norm"], 1e-5) @ d["head"].T
    device, lib = backend
    eng = SeqLMEngine(cfg, SeqLMWeights(cfg, lambda n: w[n], komazen.tensor_name, device), dtype="float32", max_tokens=32, page_size=4,
                      max_seqs=2, lib=lib)
    assert float(_rows(_prompt_then_decode(eng, toks, 4), want).max()) < 5 * TOL["float32"]


def test_greedy_generation_through_the_scheduler(backend):
    cfg = mixed_model()
    w = O.random_weights(cfg, seed=19)
    prompts = [_tokens(n, cfg["vocab"], seed=40 + n) for n in (3, 5, 1)]
    eng = make_engine(cfg, w, backend, max_seqs=2)
    outs = generate(eng, prompts, max_new_tokens=2)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for t in o:                                   # every generated token is the oracle's arg-max given what came before
            lg = O.forward(cfg, w, seq)[-1]
            top2 = lg.topk(2).values
            assert int(lg.argmax()) == t or float(top2[0] - top2[1]) < 1e-3
            seq.append(t)
        assert len(o) == 2
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
    from leopard_b200.seqlm import DenseFFConfig, LatentAttentionConfig, WindowAttentionConfig
    assert "Komazen" in registry.architectures()
    cfg = komazen.config_from_dict(mixed_model())
    assert (cfg.norm, cfg.post_alpha, cfg.embed_scale, cfg.eps) == ("post", 1.8, 1.5, 1e-5)
    a, b, c = cfg.layers
    assert all(lc.input_conv == 3 for lc in cfg.layers)
    assert isinstance(a.mixer, LatentAttentionConfig) and isinstance(a.ff, DenseFFConfig) and (a.ff.act, a.ff.ff) == ("gelu_glu", 10)
    assert (a.mixer.q_rank, a.mixer.kv_rank, a.mixer.window, a.mixer.out_gate, a.mixer.head_gate, a.mixer.kv_from, a.mixer.rot.layout) == \
        (7, 9, 5, True, False, None, "half")
    assert isinstance(b.mixer, WindowAttentionConfig) and b.ff is None
    assert (b.mixer.qk_norm, b.mixer.head_temp, b.mixer.distance_bias, b.mixer.window, b.mixer.rot.dims, b.mixer.vdim) == ("head", True, True, None, 0, 6)
    assert (c.mixer.kv_from, c.mixer.window, c.mixer.heads) == (0, 7, 3)
    assert komazen.tensor_name(3, "conv2") == "l3.canon2" and komazen.tensor_name(None, "embed") == "embed"
    with pytest.raises(ValueError):
        komazen.config_from_dict({"architecture": "other"})


@pytest.mark.parametrize("layer, key, value", [(2, "kv_from", 1), (2, "kv_from", 2), (2, "kv_rank", 8), (2, "rot", {"base": 99.0, "dims": 4})])
def test_shared_latents_must_fit(emu_lib, layer, key, value):
    """a layer that reads another's latents names an earlier latent layer with latents of its own, of the same sizes and rotation"""
    bad = mixed_model()
    bad["layers"][layer]["mixer"][key] = value
    with pytest.raises(ValueError):
        make_engine(bad, O.random_weights(bad, seed=1), ("cpu", emu_lib))


@pytest.mark.parametrize("heads, rank, rot, window", [(5, 12, 4, 7), (3, 132, 8, None), (2, 260, 4, 11), (1, 388, 12, 3), (40, 8, 0, 20)])
def test_latent_tiles_match_the_row_kernel(backend, heads, rank, rot, window):
    """latent attention by tiles of (row, head) pairs against a plain softmax over the cached rows, with a sink and a head gate: two
    requests of unequal length (one starts inside its sequence), every number of register columns, heads that straddle tiles"""
    import ctypes as C
    from leopard_b200 import _lib
    from leopard_b200.seqlm import LatentAttentionConfig, LayerConfig, RotaryConfig, SeqLMConfig, SeqLMEngine, _Batch
    device, lib = backend

    class NoWeights:
        pass
    w = NoWeights()
    w.device = torch.device(device)
    m = LatentAttentionConfig(heads=heads, dim=4, rot_dim=rot, vdim=4, kv_rank=rank, scale=0.3, rot=RotaryConfig(dims=0, base=1.0), window=window)
    eng = SeqLMEngine(SeqLMConfig("test", 5, 8, 1e-5, (LayerConfig(m, None),)), w, dtype="float32", max_tokens=96, page_size=4, max_seqs=2, lib=lib)
    g = torch.Generator().manual_seed(rank)
    lens, start = {"a": 37, "b": 5}, {"a": 6, "b": 0}
    total = {k: start[k] + lens[k] for k in lens}
    c = {k: torch.randn(total[k], rank + rot, generator=g) for k in lens}
    eng.cache.advance(eng.cache.open("a"), 0)
    eng.cache.reserve(eng.cache.get("a"), start["a"])
    eng.cache.get("a").length = start["a"]
    b = _Batch(eng, [StepEntry(k, [0] * n) for k, n in lens.items()])
    pool = eng.cache.pools[0]
    pool.fill_(float("nan"))                                      # rows nobody wrote must not be read
    for k in lens:
        pages = eng.cache.get(k).pages
        for t in range(total[k]):
            pool[pages[t // 4], t % 4] = c[k][t].to(device)
    q = torch.randn(b.R, heads * (4 + rot), generator=g).to(device)
    q_abs = (2.0 * torch.randn(b.R, heads * rank, generator=g)).to(device)
    sink, gate = torch.randn(heads, generator=g).to(device), torch.randn(b.R, heads, generator=g).to(device)
    d = _lib.LatentDesc(q=_lib.ptr(q), ldq=q.stride(0), heads=heads, dim=4, rot_dim=rot, kv_rank=rank, eps=1e-5, cache=_lib.ptr(pool), page_size=4,
                        page_table=_lib.ptr(b.page_table), max_pages=b.max_pages, window=window or 0, scale=0.3, sink=_lib.ptr(sink),
                        gate=_lib.ptr(gate), ldg=heads)
    out = torch.full((b.R, heads * rank), float("nan"), device=device)
    rc = eng.L.lp_latent_attend_tiles(C.byref(d), b.R, _lib.ptr(b.row_seq), _lib.ptr(b.row_pos), b.n_chunks, _lib.ptr(b.chunk_seq),
                                      _lib.ptr(b.chunk_row0), _lib.ptr(b.chunk_len), _lib.ptr(q_abs), q_abs.stride(0), _lib.ptr(out),
                                      out.stride(0), 1, eng._stream())
    eng._check(rc, "lp_latent_attend_tiles")
    qd, qa, r = q.cpu().double().view(b.R, heads, 4 + rot), q_abs.cpu().double().view(b.R, heads, rank), 0
    for k in lens:
        rows = c[k].double()
        for t in range(start[k], total[k]):
            lo = max(0, t - window + 1) if window else 0
            s = (qa[r] @ rows[lo:t + 1, :rank].T + qd[r, :, 4:] @ rows[lo:t + 1, rank:].T) * 0.3
            p = torch.softmax(torch.cat([s, sink.cpu().double()[:, None]], 1), 1)[:, :-1]
            want = p @ rows[lo:t + 1, :rank] * torch.sigmoid(gate.cpu().double()[r])[:, None]
            assert rel_err(out[r].view(heads, rank), want) < TOL["float32"], (k, t)
            r += 1
