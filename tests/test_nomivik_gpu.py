"""Nomivik on the GPU against the plain restatement in oracle/nomivik.py: every mechanism alone (with inputs made so that a
fault shows: a key that stands out just inside and just outside the window, scores far beyond the cap, a denominator that is
all sink, input gates that overtake the running maximum, decays that forget within a token or keep everything, a bigram
row that only one pair of tokens reaches), whole prompts with the residual stream after every layer run, prefill against
token-by-token decoding, portions, batches of unequal requests, slots released and used again, long decoding, other sizes,
and greedy generation through generate_step and the batch scheduler.  Small random configurations; none of them is a real
model's."""
import copy
import math
import types

import numpy as np
import pytest
import torch

from oracle import nomivik as O

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------------------------ configurations
def left(heads=6, kv_heads=3, dim=16, vdim=12, dims=12, base=300.0, window=19, scale=0.7, softcap=4.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
    if window:
        m["mask"] = {"size": window}
    return m


def right(heads=3, dim=10, vdim=14, gate_cap=6.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def par(lt=None, rt=None, ff=44):
    return {"type": "parallel", "mixer": {"left": lt or left(), "right": rt or right()}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def lru(width=60, blocks=3, conv=4, ff=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers=None, width=56, vocab=103, eps=1e-4, loop=(1, 4, 2), side=10, bigram=(97, 31, 5)):
    layers = layers or [lru(ff=36), par(), lru(width=44, blocks=2, conv=3), par(left(heads=4, kv_heads=4, dim=10, vdim=16, dims=6, window=37),
                                                                                 right(heads=2, dim=17, vdim=9), None), lru(conv=2)]
    c = {"architecture": "Nomivik", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    if side:
        c["token_side"] = {"dim": side}
    if bigram:
        c["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    return c


_MODELS = {}


def build(cfg, dtype="float32", seed=1):
    from mlx_vlm_b200.models.nomivik import Model, ModelConfig
    key = (repr(cfg), dtype, seed)
    if key not in _MODELS:
        W = O.random_weights(cfg, seed)
        _MODELS[key] = (Model(ModelConfig.from_dict(copy.deepcopy(cfg)), dtype=dtype).load_weights(W), W)
    return _MODELS[key]


def host(eng, t):
    eng.stream.synchronize()
    return t.detach().to("cpu", torch.float64)


def rel_rows(got, want):
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.square().mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).square().mean(-1).sqrt()


def rel(got, want):
    return rel_rows(got, want).max().item()


TOL = {"float32": 3e-5, "bfloat16": 8e-2}


def close(got, want, dtype):
    return rel(got, want) < TOL[dtype]


def tokens(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def run_alone(model, toks, cuts=None):
    """one request in its own fresh pool, its tokens cut into portions; logits of every position"""
    lm = model.language_model
    cache = lm.make_cache()
    out, at = [], 0
    for n in (cuts or [len(toks)]):
        part = toks[at:at + n]
        out.append(host(model.engine, lm.step([part], [cache], want=[list(range(len(part)))])))
        at += n
    assert at == len(toks)
    return torch.cat(out)


# ------------------------------------------------------------------------------------------------ mechanisms
def _eng(exact=True):
    from mlx_vlm_b200.layer_engine import LayerEngine
    key = "eng" if exact else "eng16"
    if key not in _MODELS:
        _MODELS[key] = LayerEngine("cuda:0", exact=exact)
    return _MODELS[key]


def dev(a, dtype=torch.float32):
    return torch.as_tensor(a).to(device="cuda:0", dtype=dtype).contiguous()


def dev16(a):
    return dev(a, torch.bfloat16)


def bf(t):
    return t.to(torch.bfloat16).to(torch.float32)


class _Pool:
    """what the mixers read of a pool: rows (caching layers, slots, capacity, row) and state (slots, floats)"""

    def __init__(self, slots=3, capacity=0, row=0, state=0, dtype=torch.float32):
        self.buf = torch.zeros((1, slots, max(capacity, 1), max(row, 1)), device="cuda:0", dtype=dtype)
        self.state = torch.full((slots, max(state, 1)), 7.0, device="cuda:0")     # stale numbers: never to be read
        torch.cuda.synchronize()


def _ctx(eng, pool, segments, eps=1e-5):
    """segments: (first row, rows, slot, first position) per sequence"""
    from mlx_vlm_b200.models.decoder_blocks import StepCtx
    T = sum(n for _, n, _, _ in segments)
    slot, pos = np.zeros(T, np.int32), np.zeros(T, np.int32)
    for a, n, s, p0 in segments:
        slot[a:a + n], pos[a:a + n] = s, np.arange(p0, p0 + n)
    return StepCtx(eng.ops, dev(slot, torch.int32), dev(pos, torch.int32), pool, eps, segments)


def _decode_ctx(eng, pool, slots, positions, eps=1e-5):
    from mlx_vlm_b200.models.decoder_blocks import StepCtx
    return StepCtx(eng.ops, dev(np.asarray(slots, np.int32), torch.int32), dev(np.asarray(positions, np.int32), torch.int32),
                   pool, eps, None)


def _walk(pool, eng, seqs, cuts, call):
    """drive a stateful op: sequence 0 in slot 2 cut into `cuts`, sequence 1 whole in slot 0 beside the second portion, then
    sequence 1 again in slot 2 (stale state).  call(ctx, rows of the step) -> outputs; returns [outputs of 0, of 1, of 1 again]"""
    a, b = seqs
    outs, at, mid = [], 0, None
    for k, cut in enumerate(cuts):
        segs = [(0, cut, 2, at)] + ([(cut, b, 0, 0)] if k == 1 else [])
        ctx = _ctx(eng, pool, segs) if (cut > 1 or k == 1) else _decode_ctx(eng, pool, [2], [at])
        y = call(ctx, [("a", at, cut)] + ([("b", 0, b)] if k == 1 else []))
        outs.append(y[:cut])
        if k == 1:
            mid = y[cut:]
        at += cut
    assert at == a
    again = call(_ctx(eng, pool, [(0, b, 2, 0)]), [("b", 0, b)])
    return torch.cat(outs), mid, again


@pytest.mark.parametrize("T", [1, 6, 70, 150])
@pytest.mark.parametrize("mul", [(31, 5), (1, 0), (0, 1), (10 ** 9 + 7, 998244353)])
def test_bigram_embedding(T, mul):
    """the pair of tokens picks the row (64-bit products), the last row for a sequence's first token, the token before a
    portion comes from the slot; the second copy, the first norm and its operand rows are the same row"""
    V, W, B = 50, 72, 41
    g = torch.Generator().manual_seed(T)
    E, Bg, nw = bf(torch.randn(V, W, generator=g)), bf(torch.randn(B + 1, W, generator=g)), bf(1 + 0.2 * torch.randn(W, generator=g))
    toks, other = tokens(T + 3, V, T), tokens(9, V, T + 1)
    cfg = {"embedding": {"bigram": {"mul_prev": mul[0], "mul_cur": mul[1], "buckets": B}}}
    w = {"embed": E.double(), "bigram": Bg.double()}
    want, want_b = O.embedding(toks, w, cfg), O.embedding(other, w, cfg)
    for exact in (True, False):
        eng = _eng(exact)
        pool = _Pool(slots=3, state=4)

        def call(ctx, parts):
            t = sum([(toks if s == "a" else other)[p:p + n] for s, p, n in parts], [])
            x, kept, xn, xb = eng.ops.embed_bigram(dev(np.asarray(t, np.int32), torch.int32), dev16(E), 1.0, dev16(Bg), mul[0], mul[1],
                                                   pool.state, ctx, keep=True, norm=dev16(nw), eps=1e-3)
            h = host(eng, x)
            assert torch.equal(h, host(eng, kept))
            n = O.rms(h, 1e-3) * nw.double()
            assert (host(eng, xn) - n).abs().max() < 1e-5
            assert (xb is None) == (exact or len(t) < 128)
            if xb is not None:
                assert torch.equal(host(eng, xb)[:, :W], host(eng, xn).float().bfloat16().double()) and host(eng, xb)[:, W:].abs().max() == 0
            return h

        got, mid, again = _walk(pool, eng, (T + 3, 9), [T, 1, 1, 1], call)
        assert (got - want).abs().max() < 1e-6 and (mid - want_b).abs().max() < 1e-6 and (again - want_b).abs().max() < 1e-6


@pytest.mark.parametrize("T,N", [(1, 40), (7, 150), (90, 63), (130, 72), (200, 1032)])
@pytest.mark.parametrize("n_branches", [0, 1, 2, 3])
def test_residual_update_of_normed_branches(T, N, n_branches):
    g = torch.Generator().manual_seed(N + n_branches)
    x, nw, extra = 3 * torch.randn(T, N, generator=g), bf(1 + 0.2 * torch.randn(N, generator=g)), torch.randn(T, N, generator=g)
    ys = [torch.randn(T, N + 4 * (N % 4 == 0), generator=g)[:, :N] * (5.0 if i else 0.01) for i in range(n_branches)]
    ws = [bf(1 + 0.3 * torch.randn(N, generator=g)) if i != 1 else None for i in range(n_branches)]
    mults = [0.5, 1.0, 0.25][:n_branches]
    for use_extra, use_norm in ((True, True), (False, True), (False, False)):
        want = x.double() + (extra.double() if use_extra else 0.0)
        for y, w, m in zip(ys, ws, mults):
            want = want + m * (y.double() if w is None else O.rms(y.double(), 1e-2) * w.double())
        for exact in (True, False):
            eng = _eng(exact)
            xd = dev(x)
            out, xb = eng.ops.close_rows(xd, [(y.to("cuda:0"), None if w is None else dev16(w), m) for y, w, m in zip(ys, ws, mults)], 1e-2,
                                         extra=dev(extra) if use_extra else None, norm=dev16(nw) if use_norm else None)
            assert (host(eng, xd) - want).abs().max() < 1e-5 * want.abs().max()
            last = want
            if use_norm:
                last = O.rms(want, 1e-2) * nw.double()
                assert (host(eng, out) - last).abs().max() < 1e-5 * last.abs().max()
            assert (xb is None) == (exact or T < 128 or N % 8 != 0)
            if xb is not None:
                xb = host(eng, xb)
                assert torch.equal(xb[:, :N], host(eng, out if use_norm else xd).float().bfloat16().double())
                assert N % 64 == 0 or xb[:, N:].abs().max() == 0


@pytest.mark.parametrize("T", [1, 3, 20, 140])
@pytest.mark.parametrize("dim,W", [(16, 64), (10, 55), (24, 200)])
def test_token_side_input(T, dim, W):
    """gate, table entry of the token (a slice of a wider table) and projection, with rows that are still to be added"""
    from mlx_vlm_b200.models.decoder_blocks import TokenSide
    V = 30
    g = torch.Generator().manual_seed(T + dim)
    w = {"side.gate": bf(torch.randn(dim, W, generator=g) / W ** 0.5), "side.proj": bf(torch.randn(W, dim, generator=g)),
         "side.norm": bf(torch.ones(W))}
    table = bf(torch.randn(V, 3 * dim, generator=g))
    x, y, tok = 2 * torch.randn(T, W, generator=g), torch.randn(T, W, generator=g), tokens(T, V, T)
    s = TokenSide(1, dim, W)
    s.bind("side.", {n: dev16(t) for n, t in w.items()}.__getitem__)
    s.table = dev16(table)[:, dim:2 * dim]
    wd = {"l1." + n: t.double() for n, t in w.items()}
    for exact in (True, False):
        eng = _eng(exact)
        ctx = _ctx(eng, None, [(0, T, 0, 0)])
        ctx.tokens = dev(np.asarray(tok, np.int32), torch.int32)
        for pending in (False, True):
            want = O.token_side(x.double() + (y.double() if pending else 0.0), table.double()[tok][:, dim:2 * dim], wd, "l1.", 1e-6)
            got = host(eng, s.rows(ctx, dev(x), pending=dev(y) if pending else None))
            assert (O.rms(got, 1e-6) - want).abs().max() < (2e-5 if exact else 0.08) * want.abs().max()


@pytest.mark.parametrize("H,G,d,dv,dims,T", [(6, 3, 16, 12, 12, 9), (4, 4, 10, 3, 10, 70), (3, 1, 40, 8, 2, 1), (2, 2, 6, 6, 0, 5), (12, 2, 96, 64, 64, 65)])
def test_unit_norms_rotation_and_cache_rows(H, G, d, dv, dims, T):
    eng = _eng()
    g = torch.Generator().manual_seed(H * d + T)
    q, k, v = 3 * torch.randn(T, H * d, generator=g), 2 * torch.randn(T, G * d, generator=g), torch.randn(T, G * dv, generator=g)
    p0, eps, rot = 90, 1e-2, {"base": 77.0, "dims": dims}
    pos = torch.arange(p0, p0 + T)
    pool = _Pool(slots=2, capacity=p0 + T, row=G * (d + dv) + 3)
    ctx = _ctx(eng, pool, [(0, T, 1, p0)], eps)
    D = dev(torch.cat([q, k, v], 1))                        # one projected row, as the product leaves it
    Q, K, V = D[:, :H * d], D[:, H * d:H * d + G * d], D[:, H * d + G * d:]
    eng.ops.head_qkv_post(Q, K, V, pool.buf[0][..., :G * (d + dv)], ctx.slot, ctx.pos, ctx.rope(77.0, dims), H, G, d, dv, dims, eps=eps,
                          unit=True)
    qr = O.rms(O.rotate_half(q.double().view(T, H, d), pos, rot), eps).reshape(T, H * d)
    kr = O.rms(O.rotate_half(k.double().view(T, G, d), pos, rot), eps).reshape(T, G * d)
    row = host(eng, pool.buf[0, 1, p0:p0 + T])
    assert (host(eng, Q) - qr).abs().max() < 3e-5 and (row[:, :G * d] - kr).abs().max() < 3e-5
    assert torch.equal(row[:, G * d:G * (d + dv)], v.double()) and row[:, G * (d + dv):].abs().max() == 0
    assert pool.buf[0, 0].abs().max() == 0


def _attend(eng, q, k, v, scale, window, n_split, softcap):
    (T, H, d), (G, dv) = q.shape, v.shape[1:]
    pool = _Pool(slots=2, capacity=T + 3, row=G * (d + dv))
    pool.buf[0, 1, :T, :G * d] = dev(k.reshape(T, G * d))
    pool.buf[0, 1, :T, G * d:] = dev(v.reshape(T, G * dv))
    slot, pos = dev(np.full(T, 1, np.int32), torch.int32), dev(np.arange(T, dtype=np.int32), torch.int32)
    out = dev(torch.zeros(T, H * dv))
    eng.ops.sink_attention(dev(q.reshape(T, H * d)), pool.buf[0], slot, pos, out, None, H, G, d, dv, scale, window=window,
                           n_split=n_split, unit_sink=True, softcap=softcap)
    return host(eng, out).view(T, H, dv)


def _attend_ref(q, k, v, scale, window, softcap):
    rep = q.shape[1] // k.shape[1]
    s = O.capped(torch.einsum("thd,shd->hts", q.double(), k.double().repeat_interleave(rep, dim=1)) * scale, softcap)
    a = O.softmax_with_one(s, O.visible(q.shape[0], window))
    return torch.einsum("hts,shd->thd", a, v.double().repeat_interleave(rep, dim=1))


@pytest.mark.parametrize("window", [1, 2, 31, 32, 33, 64, 100, 0])
@pytest.mark.parametrize("n_split", [1, 5])
def test_window_edges_cap_and_the_one_in_the_denominator(window, n_split):
    """one key far louder than the rest just inside and just outside the window of the last query; the same scores beyond a
    low cap; queries whose scores are all far below zero: the one in the denominator takes the weight"""
    eng = _eng()
    g = torch.Generator().manual_seed(window)
    H, G, d, dv, T = 4, 2, 8, 12, 140
    q, k, v = torch.randn(T, H, d, generator=g), 0.1 * torch.randn(T, G, d, generator=g), torch.randn(T, G, dv, generator=g)
    for back in ((window - 1, window) if window else (130,)):
        kk = k.clone()
        qg = q[T - 1].view(G, H // G, d)[:, 0]
        kk[T - 1 - back] = 30.0 * qg / qg.norm(dim=-1, keepdim=True)
        for cap in (0.0, 25.0, 2.0):
            got = _attend(eng, q, kk, v, 0.5, window, n_split, cap)
            assert (got - _attend_ref(q, kk, v, 0.5, window, cap)).abs().max() < 2e-5
            if cap != 2.0:
                loud = (got[T - 1, 0] - v[T - 1 - back, 0].double()).abs().max()
                assert (loud < 2e-3) == (back < window or not window)
    got = _attend(eng, torch.ones(T, H, d), -6.0 * torch.ones(T, G, d), v, 0.5, window, n_split, 25.0)
    assert got.abs().max() < 1e-6


@pytest.mark.parametrize("H,G,window,p0,n", [(4, 2, 40, 0, 300), (6, 3, 150, 70, 260), (2, 1, 128, 5, 256), (3, 3, 0, 30, 170), (8, 2, 1100, 0, 1300)])
def test_attention_of_a_long_portion_on_the_tensor_cores(H, G, window, p0, n):
    """a long portion (serving mode) through the two tensor-core products against the row kernel on the same rows, scores
    beyond the cap among them"""
    from mlx_vlm_b200.models.decoder_blocks import GroupedAttention
    eng = _eng(False)
    g = torch.Generator().manual_seed(window + n)
    m = GroupedAttention(0, left(heads=H, kv_heads=G, dim=32, vdim=24, dims=16, window=window, softcap=3.0, scale=0.5), 32, qk_norm="unit",
                         sink="unit", bias=True)
    T = p0 + n
    pool = _Pool(slots=2, capacity=T + 5, row=G * 56, dtype=torch.bfloat16)
    pool.buf[0, 1, :T] = dev(torch.randn(T, G * 56, generator=g)).to(torch.bfloat16)
    q = dev(bf(torch.randn(n, H * 32, generator=g)))
    ctx = _ctx(eng, pool, [(0, n, 1, p0)])
    a, b = dev(torch.zeros(n, H * 24)), dev(torch.zeros(n, H * 24))
    with eng.ops.on_stream():
        m._attend_prompt(ctx, q, pool.buf[0], 1, ctx.pos, a, p0, n)
        m._attend_rows(ctx, q, pool.buf[0], ctx.slot, ctx.pos, b, prompt=True)
    assert eng.ops.tc_enabled
    assert (host(eng, a) - host(eng, b)).abs().max() < 2e-3


CUTS = [[17, 1, 1, 2, 25, 84], [130], [65, 1, 63, 1], [5, 90, 2, 33], [64, 66]]


@pytest.mark.parametrize("H,d,dv", [(3, 10, 14), (1, 1, 1), (2, 32, 48), (4, 20, 7), (2, 130, 66), (1, 64, 200), (16, 16, 16), (2, 8, 96)])
@pytest.mark.parametrize("cuts", CUTS)
def test_matrix_memory_in_portions_and_slots(H, d, dv, cuts):
    """long portions (64 tokens at a time), short ones and single tokens (walked), a second sequence beside the first, a slot
    used again; input gates that overtake the running maximum late, forget gates that drop everything and that keep all"""
    eng = _eng()
    g = torch.Generator().manual_seed(H * 100 + d + len(cuts))
    cap, eps, n_b = 7.0, 1e-3, 33
    wt = bf(1 + 0.3 * torch.randn(H * dv, generator=g))

    def rand(T):
        gi, gf = 3 * torch.randn(T, H, generator=g), 3 + 3 * torch.randn(T, H, generator=g)
        gi[min(T - 1, 100):] += 25.0                        # beyond the cap
        gf[T // 3] = -40.0
        return {"q": torch.randn(T, H * d, generator=g), "k": torch.randn(T, H * d, generator=g), "v": torch.randn(T, H * dv, generator=g),
                "g": torch.randn(T, H * dv, generator=g), "gi": gi, "gf": gf}

    data = {"a": rand(130), "b": rand(n_b)}

    def ref(x):
        T = x["q"].shape[0]
        r = {k: t.double() for k, t in x.items()}
        i, f = O.capped(r["gi"], cap), torch.nn.functional.logsigmoid(O.capped(r["gf"], cap))
        o = O.memory_walk(r["q"].view(T, H, d) * d ** -0.5, r["k"].view(T, H, d), r["v"].view(T, H, dv), i, f)
        return O.rms(o, eps).reshape(T, H * dv) * wt.double() * torch.sigmoid(r["g"])

    from mlx_vlm_b200.models.decoder_blocks import MatrixMemory
    n_state = MatrixMemory(0, right(H, d, dv), 8).state_floats
    pool = _Pool(slots=3, state=4 + n_state)
    st = pool.state[:, 4:]

    def call(ctx, parts):
        x = {k: torch.cat([data[s][k][p:p + n] for s, p, n in parts]) for k in data["a"]}
        D = dev(torch.cat([x[k] for k in ("q", "k", "v", "g", "gi", "gf")], 1))
        at, c = 0, {}
        for k in ("q", "k", "v", "g", "gi", "gf"):
            c[k] = D[:, at:at + x[k].shape[1]]
            at += x[k].shape[1]
        return host(eng, eng.ops.matrix_memory(c["q"], c["k"], c["v"], c["gi"], c["gf"], c["g"], dev16(wt), st, ctx, H=H, dim=d, vdim=dv,
                                               cap=cap, q_scale=float(d) ** -0.5, eps=eps))

    got, mid, again = _walk(pool, eng, (130, n_b), cuts if len(cuts) > 1 else [129, 1], call)
    wa, wb = ref(data["a"]), ref(data["b"])
    tol = 1e-4 * max(1.0, wa.abs().max().item())
    assert (got - wa).abs().max() < tol and (mid - wb).abs().max() < tol and (again - wb).abs().max() < tol


def test_matrix_memory_operand_rows_and_recall():
    """a key stored 190 tokens ago comes back when the forget gates keep everything; bf16 operand rows are the rounded rows"""
    eng = _eng(False)
    T, H, d, dv = 200, 1, 8, 5
    q, k, v = torch.zeros(T, d), torch.zeros(T, d), torch.zeros(T, dv)
    k[9, 2] = 4.0
    v[9] = torch.tensor([1.0, 2.0, 3.0, 4.0, 5.0])
    q[T - 1, 2] = 4.0
    pool = _Pool(slots=1, state=64)
    args = lambda: (dev(q), dev(k), dev(v), dev(torch.zeros(T, 1)), dev(torch.full((T, 1), 60.0)), dev(torch.full((T, dv), 40.0)),
                    dev16(torch.ones(dv)), pool.state, _ctx(eng, pool, [(0, T, 0, 0)]))
    kw = dict(H=H, dim=d, vdim=dv, cap=30.0, q_scale=1.0, eps=1e-9)
    y = host(eng, eng.ops.matrix_memory(*args(), **kw))
    want = v[9].double() / v[9].double().square().mean().sqrt()
    assert (y[T - 1] - want).abs().max() < 1e-5 and y[:T - 1].abs().max() == 0
    yb = host(eng, eng.ops.matrix_memory(*args(), operand=True, **kw))
    assert torch.equal(yb[:, :dv], y.float().bfloat16().double()) and yb[:, dv:].abs().max() == 0


@pytest.mark.parametrize("n,nb", [(60, 3), (44, 44), (130, 1), (256, 2), (1, 1)])
@pytest.mark.parametrize("cuts", CUTS)
def test_gated_recurrence_in_portions_and_slots(n, nb, cuts):
    """long portions (in parts), short ones and single tokens; decays from one token to thousands, gates that close"""
    eng = _eng()
    g = torch.Generator().manual_seed(n + len(cuts))
    bs, n_b = n // nb, 33
    rb, ib, lam = bf(2 * torch.randn(n, generator=g)), bf(torch.randn(n, generator=g)), bf(-6 + 5 * torch.randn(n, generator=g))

    def rand(T):
        return {"G": 3 * torch.randn(T, 2 * n, generator=g), "u": torch.randn(T, n, generator=g), "y": 2 * torch.randn(T, n, generator=g)}

    data = {"a": rand(130), "b": rand(n_b)}

    def ref(x):
        G = x["G"].double().view(-1, nb, 2, bs)
        r = torch.sigmoid(G[:, :, 0].reshape(-1, n) + rb.double())
        i = torch.sigmoid(G[:, :, 1].reshape(-1, n) + ib.double())
        return O.recurrence(x["u"].double(), r, i, lam.double()) * O.gelu(x["y"].double())

    for operand in (False, True):
        pool = _Pool(slots=3, state=n + 3)
        st = pool.state[:, 3:]

        def call(ctx, parts):
            x = {k: torch.cat([data[s][k][p:p + m] for s, p, m in parts]) for k in data["a"]}
            yu = dev(torch.cat([x["y"], x["u"]], 1))
            y = host(eng, eng.ops.gated_recurrence(dev(x["G"]), bs, dev16(rb), dev16(ib), dev16(lam), 8.0, yu[:, n:], yu[:, :n], st, ctx,
                                                   operand=operand))
            assert not operand or y.shape[1] == n or y[:, n:].abs().max() == 0
            return y[:, :n]

        got, mid, again = _walk(pool, eng, (130, n_b), cuts if len(cuts) > 1 else [129, 1], call)
        wa, wb = ref(data["a"]), ref(data["b"])
        tol = 2e-5 * wa.abs().max()
        if operand:
            assert ((got - wa).abs() <= wa.abs() / 128 + tol).all() and ((again - wb).abs() <= wb.abs() / 128 + tol).all()
        else:
            assert (got - wa).abs().max() < tol and (mid - wb).abs().max() < tol and (again - wb).abs().max() < tol


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_convolution_in_portions_and_slots(taps):
    eng = _eng()
    g = torch.Generator().manual_seed(taps)
    C = 70
    c, b = bf(torch.randn(C, taps, generator=g)), bf(torch.randn(C, generator=g))
    data = {"a": torch.randn(130, C, generator=g), "b": torch.randn(33, C, generator=g)}
    for cuts in CUTS:
        pool = _Pool(slots=3, state=(taps - 1) * C + 5)
        st = pool.state[:, 2:2 + (taps - 1) * C]

        def call(ctx, parts):
            return host(eng, eng.ops.short_conv(dev(torch.cat([data[s][p:p + n] for s, p, n in parts])), dev16(c), st, ctx, bias=dev16(b)))

        got, mid, again = _walk(pool, eng, (130, 33), cuts if len(cuts) > 1 else [129, 1], call)
        wa, wb = (O.conv(data[s].double(), c.double(), b.double()) for s in "ab")
        assert (got - wa).abs().max() < 1e-5 and (mid - wb).abs().max() < 1e-5 and (again - wb).abs().max() < 1e-5


@pytest.mark.parametrize("n,nb,T", [(60, 3, 5), (60, 3, 40), (128, 2, 150), (192, 3, 300), (96, 4, 150), (50, 5, 150)])
def test_gate_logits_of_the_blocks(n, nb, T):
    """both gates of every block in one product; the serving mode's long steps keep more of u than one bf16 part"""
    from mlx_vlm_b200.models.decoder_blocks import GatedRecurrence
    g = torch.Generator().manual_seed(n + T)
    bs = n // nb
    m = GatedRecurrence(0, {"width": n, "blocks": nb, "conv": 4}, 32)
    ra, ri = (bf(torch.randn(nb, bs, bs, generator=g) / bs ** 0.5) for _ in range(2))
    m.w = {"gates": dev16(torch.cat([ra, ri], 1))}
    u = 2 * torch.randn(T, n, generator=g)
    zero = torch.zeros(nb, bs, dtype=torch.float64)
    want = torch.stack([O.block_linear(u.double(), w.double(), zero).view(T, nb, bs) for w in (ra, ri)], 2).reshape(T, 2 * n)
    for exact in (True, False):
        eng = _eng(exact)
        assert (host(eng, m._gate_logits(eng.ops, dev(u))) - want).abs().max() < 2e-4
        assert eng.ops.tc_enabled


# ------------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt_and_every_layer_run(dtype):
    cfg = config()
    model, W = build(cfg, dtype)
    toks = tokens(150, cfg["vocab"], 1)
    ref, layers_ref = O.forward(cfg, W, toks, return_layers=True)
    assert close(run_alone(model, toks), ref, dtype)
    if dtype == "float32":
        eng, lm = model.engine, model.language_model
        seen = []
        real = [L.forward for L in model.layers]
        try:
            for L, f in zip(model.layers, real):
                def wrapped(c, xx, *a, f=f, **kw):
                    out = f(c, xx, *a, **kw)
                    extra = kw.get("extra")        # what comes ahead of the next pass rides in the same launch
                    seen.append(host(eng, xx) - (0.0 if extra is None else host(eng, extra)))
                    return out
                L.forward = wrapped
            lm.step([toks], [lm.make_cache()])
        finally:
            for L, f in zip(model.layers, real):
                L.forward = f
        assert len(seen) == len(layers_ref) == 8
        for got, want in zip(seen, layers_ref):
            assert (got - want).abs().max() < 3e-5 * max(1.0, want.abs().max().item())


def test_first_tokens():
    cfg = config()
    model, W = build(cfg)
    for n in (1, 2, 3, 4, 5):
        toks = tokens(n, cfg["vocab"], 10 + n)
        assert rel(run_alone(model, toks), O.forward(cfg, W, toks)) < TOL["float32"]
        assert rel(run_alone(model, toks, [1] * n), O.forward(cfg, W, toks)) < TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_then_token_by_token(dtype):
    cfg = config()
    model, W = build(cfg, dtype)
    toks = tokens(110, cfg["vocab"], 2)
    ref = O.forward(cfg, W, toks)
    got = run_alone(model, toks, [50] + [1] * 60)       # every window passes over decoded tokens
    assert close(got, ref, dtype)
    if dtype == "float32":
        assert rel(got, run_alone(model, toks)) < TOL[dtype]


@pytest.mark.parametrize("cuts", [[2] * 35, [3, 64, 3], [31, 1, 32, 6], [18, 1, 19, 20, 12], [69, 1], [17, 17, 36], [65, 5]])
def test_portions(cuts):
    cfg = config()
    model, W = build(cfg)
    toks = tokens(70, cfg["vocab"], 3)
    assert rel(run_alone(model, toks, cuts), O.forward(cfg, W, toks)) < TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone(dtype):
    cfg = config()
    model, W = build(cfg, dtype)
    lm, eng = model.language_model, model.engine
    lens = [1, 45, 130, 18]
    reqs = [tokens(n + 12, cfg["vocab"], 20 + n) for n in lens]
    pool = lm.make_pool(4, 64)                       # too short on purpose: it grows under the batch
    caches = [lm.make_cache_row(pool, s) for s in (2, 0, 3, 1)]
    first = host(eng, lm.step([r[:n] for r, n in zip(reqs, lens)], caches, want=[list(range(n)) for n in lens]))
    got = list(torch.split(first, lens))
    for k in range(12):                              # then all go on by one token, together
        step = host(eng, lm.step([[r[n + k]] for r, n in zip(reqs, lens)], caches))
        got = [torch.cat([g, step[i:i + 1]]) for i, g in enumerate(got)]
    for g, r in zip(got, reqs):
        assert close(g, O.forward(cfg, W, r), dtype)
        if dtype == "float32":
            assert rel(g, run_alone(model, r)) < TOL[dtype]


def test_many_single_tokens_in_one_step():
    """more requests in a decode step than the few-rows kernels take"""
    cfg = config()
    model, W = build(cfg)
    lm, eng = model.language_model, model.engine
    pool = lm.make_pool(20, 32)
    reqs = [tokens(5 + i % 4, cfg["vocab"], 300 + i) for i in range(20)]
    caches = [lm.make_cache_row(pool, s) for s in range(20)]
    lm.step([r[:-1] for r in reqs], caches)
    got = host(eng, lm.step([[r[-1]] for r in reqs], caches))
    for i, r in enumerate(reqs):
        assert rel(got[i:i + 1], O.forward(cfg, W, r)[-1:]) < TOL["float32"]


def test_slots_released_and_used_again_and_more_slots():
    from mlx_vlm_b200.models.cache import SlotTable
    cfg = config()
    model, W = build(cfg)
    lm, eng = model.language_model, model.engine
    pool, table = lm.make_pool(2, 64), SlotTable(2)
    a, b, c, d = (tokens(n, cfg["vocab"], 40 + n) for n in (40, 25, 33, 50))
    ca, cb = lm.make_cache_row(pool, table.acquire("a")), lm.make_cache_row(pool, table.acquire("b"))
    lm.step([a[:30], b], [ca, cb])
    table.release("b")                                   # b is finished; c takes its slot (and b's stale rows and state)
    cc = lm.make_cache_row(pool, table.acquire("c"))
    assert cc[0]._row == 1 and cc[0].offset == 0 and not cc[0].is_trimmable()
    got = host(eng, lm.step([a[30:], c], [ca, cc], want=[list(range(10)), list(range(33))]))
    assert rel(got[:10], O.forward(cfg, W, a)[30:]) < TOL["float32"]
    assert rel(got[10:], O.forward(cfg, W, c)) < TOL["float32"]
    with torch.cuda.stream(eng.stream):                  # a third live request: the pool gets more slots
        pool.add_slots(4, live_tokens=pool.capacity)
    table.grow(4)
    cd = lm.make_cache_row(pool, table.acquire("d"))
    assert cd[0]._row == 2
    got = host(eng, lm.step([[a[0]], d], [ca, cd], want=[[], list(range(50))]))
    assert rel(got, O.forward(cfg, W, d)) < TOL["float32"]
    got = host(eng, lm.step([[5]], [cc]))                # c's rows, state and last token survived the move
    assert rel(got, O.forward(cfg, W, c + [5])[-1:]) < TOL["float32"]
    eng.kv_copy_row(pool, 3, pool, 1, cc[0].offset)      # a slot copied to another row (the scheduler's compaction)
    moved = lm.make_cache_row(pool, 3)
    for m in moved:
        m.offset = cc[0].offset
    got = host(eng, lm.step([[9]], [moved]))
    assert rel(got, O.forward(cfg, W, c + [5, 9])[-1:]) < TOL["float32"]


def test_long_prompt_paths_of_the_serving_mode():
    """prompts of 128 tokens and more take the tensor-core products (projections, gates of whole and of ragged blocks,
    attention in chunks, the token input); a long portion after a cached prefix; a batch whose short member stays on the row
    kernels"""
    cfg = config([par(left(heads=4, kv_heads=2, dim=24, vdim=16, dims=16, window=40), right(heads=2, dim=16, vdim=24), 48),
                  lru(width=128, blocks=2, conv=4, ff=40), lru(width=96, blocks=4, conv=2),
                  par(left(heads=2, kv_heads=1, dim=16, vdim=16, dims=8, window=150), right(heads=4, dim=8, vdim=8), None)],
                 width=64, loop=(0, 2, 2), side=16)
    model, W = build(cfg, "bfloat16", seed=4)
    exact, _ = build(cfg, "float32", seed=4)
    lm, eng = model.language_model, model.engine
    toks = tokens(400, cfg["vocab"], 9)
    ref = O.forward(cfg, W, toks)
    assert close(run_alone(model, toks), ref, "bfloat16")
    assert close(run_alone(model, toks, [140, 220, 40]), ref, "bfloat16")
    assert rel(run_alone(exact, toks, [140, 220, 40]), ref) < TOL["float32"]
    assert model.engine.ops.tc_enabled
    pool = lm.make_pool(2, 512)
    ca, cb = lm.make_cache_row(pool, 0), lm.make_cache_row(pool, 1)
    both = host(eng, lm.step([toks[:200], toks[:30]], [ca, cb], want=[list(range(200)), list(range(30))]))
    assert close(both[:200], ref[:200], "bfloat16") and close(both[200:], ref[:30], "bfloat16")


def test_row_kernels_take_over_when_the_tensor_cores_refuse():
    cfg = config([par(left(heads=4, kv_heads=2, dim=24, vdim=16, dims=16, window=40), right(heads=2, dim=16, vdim=24), 48),
                  lru(width=128, blocks=2, conv=4, ff=40)], width=64, loop=None, side=16)
    W = O.random_weights(cfg, 6)
    from mlx_vlm_b200._native import B200Error
    from mlx_vlm_b200.models.nomivik import Model, ModelConfig
    toks = tokens(160, cfg["vocab"], 9)
    ref = O.forward(cfg, W, toks)
    for at in (0, 3, 7, 12):                             # the product that is refused: each leaves another step half done
        model = Model(ModelConfig.from_dict(copy.deepcopy(cfg)), dtype="bfloat16").load_weights(W)
        ops, seen = model.engine.ops, [0]
        real = ops.tc_gemm

        def refuse(*a, **kw):
            seen[0] += 1
            if seen[0] > at:
                raise B200Error("refused")
            return real(*a, **kw)

        ops.tc_gemm = refuse
        assert close(run_alone(model, toks), ref, "bfloat16") and not ops.tc_enabled


def test_long_decoding():
    cfg = config()
    model, W = build(cfg)
    toks = tokens(330, cfg["vocab"], 5)
    got = run_alone(model, toks, [20] + [1] * 310)
    assert rel(got, O.forward(cfg, W, toks)) < TOL["float32"]


OTHER = {
    "no loop, no token input, no bigram": config([par(), lru(ff=20)], loop=None, side=0, bigram=None),
    "a loop without a bigram, three passes of one layer": config([lru(width=30, blocks=1, ff=16), par(ff=None)], loop=(1, 2, 3), bigram=None),
    "one pass of the span": config([par(ff=20), lru()], loop=(0, 2, 1), side=3),
    "attention layers only, equal sizes": config([par(left(heads=4, kv_heads=4, dim=8, vdim=8, dims=8, window=5), right(heads=4, dim=8, vdim=8), 32),
                                                  par(left(heads=4, kv_heads=4, dim=8, vdim=8, dims=8, window=5), right(heads=4, dim=8, vdim=8), 32)],
                                                 width=32, loop=(0, 1, 2), side=32, vocab=32),
    "recurrences only, one block, one channel each": config([lru(width=7, blocks=1, conv=1, ff=9), lru(width=12, blocks=12, conv=6)], loop=(0, 2, 2),
                                                            width=40, vocab=37, side=1, bigram=(1, 1, 1)),
    "one head, a window of one, sizes of one": config([par(left(heads=1, kv_heads=1, dim=2, vdim=1, dims=2, window=1, scale=1.0, softcap=1.0),
                                                           right(heads=1, dim=1, vdim=1, gate_cap=1.0), 1), lru(width=1, blocks=1, conv=4)],
                                                      loop=(1, 2, 2), width=24, vocab=19, side=2),
    "no window, no rotation, no cap, wide heads": config([par(left(heads=3, kv_heads=1, dim=72, vdim=40, dims=0, window=0, softcap=None),
                                                              right(heads=2, dim=72, vdim=136, gate_cap=15.0), 30), lru(width=72, blocks=2)],
                                                         width=72, vocab=257, loop=(0, 2, 2), bigram=(1000, 7, 1)),
    "the span at the end, rotated to the last number, odd sizes": config(
        [lru(width=33, blocks=3, conv=5, ff=21), par(left(heads=10, kv_heads=5, dim=6, vdim=7, dims=6, window=64), right(heads=5, dim=3, vdim=11), 27)],
        width=45, vocab=61, loop=(1, 2, 4), side=5, eps=1e-6),
}


@pytest.mark.parametrize("name", sorted(OTHER))
def test_other_sizes(name):
    cfg = OTHER[name]
    model, W = build(cfg, seed=7)
    toks = tokens(75, cfg["vocab"], 6)
    ref = O.forward(cfg, W, toks)
    assert rel(run_alone(model, toks), ref) < TOL["float32"]
    assert rel(run_alone(model, toks, [40] + [1] * 35), ref) < TOL["float32"]
    assert rel(run_alone(model, toks, [7, 2, 66]), ref) < TOL["float32"]
    served, _ = build(cfg, "bfloat16", seed=7)
    assert close(run_alone(served, toks, [40] + [1] * 35), ref, "bfloat16")


# ------------------------------------------------------------------------------------------------ generation
def oracle_greedy(cfg, W, prompt, n):
    toks, margins = list(prompt), []
    for _ in range(n):
        z = O.forward(cfg, W, toks)[-1]
        top2 = torch.topk(z, 2).values
        margins.append(float(top2[0] - top2[1]))
        toks.append(int(torch.argmax(z)))
    return toks[len(prompt):], margins


def same_until_tie(got, want, margins, what):
    for i, (g, w) in enumerate(zip(got, want)):
        if margins[i] < 1e-3:
            return
        assert g == w, f"{what}: token {i} is {g}, the plain implementation says {w}"


def test_greedy_generate_step():
    from mlx_vlm_b200.generate import generate_step
    cfg = config()
    model, W = build(cfg)
    prompt = tokens(21, cfg["vocab"], 8)
    want, margins = oracle_greedy(cfg, W, prompt, 20)       # past two eager steps the step is a replayed graph
    got = [t for t, _ in generate_step(np.asarray([prompt]), model, None, None, max_tokens=20)]
    same_until_tie(got, want, margins, "generate_step")
    assert model.engine.graph_replays > 0
    got = [t for t, _ in generate_step(np.asarray([prompt]), model, None, None, max_tokens=8, prefill_step_size=6)]
    same_until_tie(got, want[:8], margins, "generate_step with the prompt in portions")
    from mlx_vlm_b200.sample_utils import make_sampler
    got = [t for t, _ in generate_step(np.asarray([prompt]), model, None, None, max_tokens=6,
                                       sampler=make_sampler(temp=0.0), logit_bias={0: 0.0})]
    same_until_tie(got, want[:6], margins, "generate_step with a sampler")
    emb = model.get_input_embeddings(np.asarray([prompt])).inputs_embeds
    w = {k: t.double() for k, t in W.items()}
    assert (host(model.engine, emb)[0] - O.embedding(prompt, w, cfg)).abs().max() < 1e-6


def test_batch_scheduler_lock_step_rows():
    from mlx_vlm_b200.generate_batch import BatchGenerator
    cfg = config()
    model, W = build(cfg)
    model.config.eos_token_id = []
    prompts = [tokens(n, cfg["vocab"], 60 + n) for n in (5, 30, 12, 44, 9)]
    n_new = [6, 9, 4, 7, 5]
    proc = types.SimpleNamespace(tokenizer=types.SimpleNamespace(stopping_criteria=None))
    g = BatchGenerator(model, proc, completion_batch_size=3, prefill_batch_size=2, decode_slice=2)
    uids = g.insert(prompts, n_new)
    out = {u: [] for u in uids}
    while g.has_work:
        for r in g.next()[1]:
            out[r.uid].append(r.token)
    for u, p, n in zip(uids, prompts, n_new):
        want, margins = oracle_greedy(cfg, W, p, n)
        assert len(out[u]) == n
        same_until_tie(out[u], want, margins, f"row {u}")


def test_trace_runner_from_a_checkpoint_folder(tmp_path):
    """bin/trace_run on a checkpoint folder: the registry picks the class from `architecture`, requests are prefilled
    together, decoded together, one ends and a later one takes its slot; both number formats"""
    import json
    import os
    import subprocess
    import sys
    from safetensors.torch import save_file
    cfg = config()
    W = O.random_weights(cfg, 11)
    model_dir = tmp_path / "model"
    model_dir.mkdir()
    (model_dir / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in W.items()}, str(model_dir / "model.safetensors"))
    a, b, c = (tokens(n, cfg["vocab"], 70 + n) for n in (40, 9, 25))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:8], "want": [7]}],
              "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:31], "want": [0]}, {"id": "b", "tokens": b[8:], "want": [0]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[31:32], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[32:], "want": [7]}, {"id": "c", "tokens": c, "want": [0, 24]}],
              "end": ["a", "c"]}]
    want = {0: [(a, 0), (a, 29), (b, 7)], 1: [(a, 30), (b, 8)], 3: [(a, 39), (c, 0), (c, 24)]}
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype in ("bfloat16", "float32"):
        out = tmp_path / dtype
        r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(model_dir), "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "80"], input="".join(json.dumps(x) + "\n" for x in steps),
                           capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
        assert not (out / "2.f32").exists()
        for st, rows in want.items():
            got = torch.from_numpy(np.fromfile(out / f"{st}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"])).double()
            ref = torch.stack([O.forward(cfg, W, t)[i] for t, i in rows])
            assert close(got, ref, dtype)
