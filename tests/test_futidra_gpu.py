"""Futidra on the GPU against the plain restatement in oracle/futidra.py: every mechanism alone (with inputs made so that a
fault shows: a key that stands out just inside and just outside the window, at a staging tile's edge and far back; a
sink that takes everything; a state whose channels forget at once or never; decays of very different strength within
one chunk), whole prompts with the residual stream after every layer, prefill against token-by-token decoding,
portions, batches of unequal requests, slots released and used again, long decoding, other sizes, and greedy
generation through generate_step and the batch scheduler.  Small random configurations; none of them is a real
model's."""
import copy
import math
import types

import numpy as np
import pytest
import torch

from oracle import futidra as O

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------------------------ configurations
def att(heads=6, kv_heads=3, dim=16, dims=12, base=400.0, scaling=(5.0, 1.0, 6.0, 64), window=19, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if window:
        m["mask"] = {"size": window}
    return m


def lat(heads=5, dim=12, vdim=10, kv_rank=28, q_rank=20, window=11, kv_from=None, scale=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def delta(heads=4, kv_heads=2, dim=20, vdim=14, conv=3, **kw):
    return dict({"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, **kw)


def layer(kind, mixer, ff=44):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers=None, width=56, vocab=103, eps=1e-5, alpha=1.6):
    layers = layers or [layer("latent_attention", lat()), layer("channel_delta", delta(), None), layer("attention", att()),
                        layer("latent_attention", lat(heads=3, dim=8, vdim=16, q_rank=12, window=37, kv_from=0), 30),
                        layer("channel_delta", delta(heads=2, kv_heads=2, dim=9, vdim=21, conv=2), 52)]
    return {"architecture": "Futidra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "postln_alpha": alpha}


_MODELS = {}


def build(cfg, dtype="float32", seed=1):
    from mlx_vlm_b200.models.futidra import Model, ModelConfig
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


@pytest.mark.parametrize("T,N", [(1, 40), (7, 150), (90, 64), (130, 72), (200, 1032)])
def test_norm_of_the_sum(T, N):
    """x <- LN(a x + y) w + b in place, rows with a large mean; in a long step of the serving mode also as bf16 operand
    rows; the model's norm with a bias over gathered rows"""
    g = torch.Generator().manual_seed(N)
    x, y = 3.0 * torch.randn(T, N, generator=g) + 20.0, torch.randn(T, N, generator=g) * torch.linspace(0.1, 9.0, N)
    w, b = bf(1 + 0.2 * torch.randn(N, generator=g)), bf(torch.randn(N, generator=g))
    want = O.post_norm(x.double(), y.double(), 1.7, w.double(), b.double(), 1e-3)
    for exact in (True, False):
        eng = _eng(exact)
        xd = dev(x)
        xb = eng.ops.sum_norm_rows(dev(y), xd, dev(w, torch.bfloat16), dev(b, torch.bfloat16), 1e-3, keep=1.7, center=True)
        got = host(eng, xd)
        assert (got - want).abs().max() < 2e-5 * want.abs().max()
        assert (xb is None) == (exact or T < 128)
        if xb is not None:
            xb = host(eng, xb)
            assert xb.shape[1] == (N + 63) // 64 * 64 and xb[:, N:].abs().max() == 0 if N % 64 else xb.shape[1] == N
            assert torch.equal(xb[:, :N], got.float().bfloat16().double())
    eng = _eng()
    rows = dev(np.asarray([T - 1, 0], np.int32), torch.int32)
    out = dev(torch.zeros(2, N))
    eng.ops.norm_rows(dev(x), dev(w, torch.bfloat16), 1e-3, out, center=True, rows=rows, bias=dev(b, torch.bfloat16))
    want = O.layer_norm(x.double(), w.double(), b.double(), 1e-3)[[T - 1, 0]]
    assert (host(eng, out) - want).abs().max() < 2e-5 * want.abs().max()


@pytest.mark.parametrize("base,dims,scaling", [(10000.0, 16, (8.0, 1.0, 4.0, 8192)), (50.0, 10, (3.0, 2.0, 5.0, 64)),
                                               (1e6, 64, (32.0, 1.0, 8.0, 100)), (300.0, 12, None)])
def test_frequencies_scaled_by_wavelength(base, dims, scaling):
    eng = _eng()
    sc = None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))
    from mlx_vlm_b200.models.layer_ops import WAVELENGTH
    key = None if scaling is None else (WAVELENGTH, scaling[0], float(scaling[3]), scaling[1], scaling[2])
    got = host(eng, eng.ops.inv_freq(base, dims, key))
    want = torch.tensor(O.frequencies(base, dims, sc), dtype=torch.float64)
    assert ((got - want).abs() / want).max() < 1e-12
    cs = host(eng, eng.ops.rope_table(dev(np.asarray([0, 3, 70001], np.int32), torch.int32), base, dims, key))
    assert (cs[2, :, 0] - torch.cos(70001.0 * want)).abs().max() < 1e-6           # angles far out stay exact, amplitude one


@pytest.mark.parametrize("pairs", [True, False])
@pytest.mark.parametrize("norm", [True, False])
@pytest.mark.parametrize("H,G,d,dims,T", [(6, 3, 16, 12, 9), (4, 4, 10, 10, 70), (3, 1, 40, 2, 1), (2, 2, 6, 0, 5), (12, 2, 96, 64, 65)])
def test_per_head_projection_post(pairs, norm, H, G, d, dims, T):
    """norm per head with one weight, rotation, keys and raw keys-as-values into the cache rows: nothing beside them moves"""
    eng = _eng()
    g = torch.Generator().manual_seed(H * d + T)
    q, k = 3 * torch.randn(T, H * d, generator=g), 2 * torch.randn(T, G * d, generator=g)
    qw, kw = bf(1 + 0.3 * torch.randn(d, generator=g)), bf(1 + 0.3 * torch.randn(d, generator=g))
    p0, eps = 90, 1e-3
    rot = {"base": 77.0, "dims": dims, "scaling": {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 30}}
    pos = torch.arange(p0, p0 + T)
    pool = _Pool(slots=2, capacity=p0 + T, row=2 * G * d + 3)
    ctx = _ctx(eng, pool, [(0, T, 1, p0)], eps)
    from mlx_vlm_b200.models.layer_ops import WAVELENGTH
    both = dev(torch.cat([q, k], 1))                        # one projected row, as the product leaves it
    Q, K = both[:, :H * d], both[:, H * d:]
    eng.ops.head_qkv_post(Q, K, K, pool.buf[0][..., :2 * G * d], ctx.slot, ctx.pos,
                          ctx.rope(77.0, dims, (WAVELENGTH, 3.0, 30.0, 1.0, 4.0)), H, G, d, d, dims, pairs=pairs, eps=eps,
                          q_norm=dev(qw, torch.bfloat16) if norm else None, k_norm=dev(kw, torch.bfloat16) if norm else None)
    qr, kr = q.double().view(T, H, d), k.double().view(T, G, d)
    if norm:
        qr, kr = O.rms(qr, eps) * qw.double(), O.rms(kr, eps) * kw.double()

    def turn(v):
        if pairs or dims < 2:
            return O.rotate_pairs(v, pos, rot)
        perm = [j for i in range(dims // 2) for j in (i, i + dims // 2)] + list(range(dims, d))    # halves as pairs
        out = torch.empty_like(v)
        out[..., perm] = O.rotate_pairs(v[..., perm], pos, rot)
        return out

    row = host(eng, pool.buf[0, 1, p0:p0 + T])
    assert (host(eng, Q) - turn(qr).reshape(T, H * d)).abs().max() < 3e-5
    assert (row[:, :G * d] - turn(kr).reshape(T, G * d)).abs().max() < 3e-5
    assert torch.equal(row[:, G * d:2 * G * d], k.double()) and row[:, 2 * G * d:].abs().max() == 0
    assert torch.equal(host(eng, K), k.double()) and pool.buf[0, 0].abs().max() == 0


def _attend(eng, q, k, v, H, G, d, scale, window, n_split):
    ops, T = eng.ops, q.shape[0]
    pool = _Pool(slots=2, capacity=T + 3, row=2 * G * d)
    pool.buf[0, 1, :T, :G * d] = dev(k.reshape(T, G * d))
    pool.buf[0, 1, :T, G * d:] = dev(v.reshape(T, G * d))
    slot, pos = dev(np.full(T, 1, np.int32), torch.int32), dev(np.arange(T, dtype=np.int32), torch.int32)
    out = dev(torch.zeros(T, H * d))
    ops.sink_attention(dev(q.reshape(T, H * d)), pool.buf[0], slot, pos, out, None, H, G, d, d, scale, window=window,
                       n_split=n_split, unit_sink=True)
    return host(eng, out).view(T, H, d)


@pytest.mark.parametrize("window", [1, 2, 31, 32, 33, 64, 100, 0])
@pytest.mark.parametrize("n_split", [1, 5])
def test_window_edges_and_the_one_in_the_denominator(window, n_split):
    """one key far louder than the rest just inside and just outside the window of the last query (and far back without
    a window); queries whose scores are all far below zero: the one in the denominator takes the weight"""
    eng = _eng()
    g = torch.Generator().manual_seed(window)
    H, G, d, T = 4, 2, 8, 140
    q, k, v = torch.randn(T, H, d, generator=g), 0.1 * torch.randn(T, G, d, generator=g), torch.randn(T, G, d, generator=g)
    for back in ((window - 1, window) if window else (130,)):
        kk = k.clone()
        qg = q[T - 1].view(G, H // G, d)[:, 0]
        kk[T - 1 - back] = 30.0 * qg / qg.norm(dim=-1, keepdim=True)
        got = _attend(eng, q, kk, v, H, G, d, 0.5, window, n_split)
        s = torch.einsum("thd,shd->hts", q.double(), kk.double().repeat_interleave(H // G, dim=1)) * 0.5
        a = O.softmax(s, O.visible(T, window), True)
        want = torch.einsum("hts,shd->thd", a, v.double().repeat_interleave(H // G, dim=1))
        assert (got - want).abs().max() < 2e-5
        loud = (got[T - 1, 0] - v[T - 1 - back, 0].double()).abs().max()
        assert (loud < 1e-3) == (back < window or not window)
    low = torch.ones(T, G, d) * -6.0
    got = _attend(eng, torch.ones(T, H, d), low, v, H, G, d, 0.5, window, n_split)
    assert got.abs().max() < 1e-6


@pytest.mark.parametrize("window", [1, 2, 32, 33, 70, 0])
@pytest.mark.parametrize("n_split", [1, 4])
def test_latent_rows_without_positions_window_and_gate(window, n_split):
    """the absorbed attention over latent rows alone, a loud latent just inside and just outside the window"""
    eng = _eng()
    g = torch.Generator().manual_seed(window + 9)
    H, r, T = 5, 24, 120
    q, c = torch.randn(T, H, r, generator=g), 0.1 * torch.randn(T, r, generator=g)
    for back in ((window - 1, window) if window else (110,)):
        cc = c.clone()
        cc[T - 1 - back] = 40.0 * q[T - 1, 2] / q[T - 1, 2].norm()
        pool = _Pool(slots=2, capacity=T, row=r)
        pool.buf[0, 1] = dev(cc)
        slot, pos = dev(np.full(T, 1, np.int32), torch.int32), dev(np.arange(T, dtype=np.int32), torch.int32)
        out = dev(torch.zeros(T, H * r))
        eng.ops.latent_attention(dev(q.reshape(T, H * r)), pool.buf[0], slot, pos, out, H, r, 0.4, window=window, n_split=n_split)
        a = O.softmax(torch.einsum("thd,sd->hts", q.double(), cc.double()) * 0.4, O.visible(T, window), False)
        want = torch.einsum("hts,sd->thd", a, cc.double())
        assert (host(eng, out).view(T, H, r) - want).abs().max() < 5e-5
        assert ((host(eng, out).view(T, H, r)[T - 1, 2] - cc[T - 1 - back].double()).abs().max() < 1e-3) == (back < window or not window)
    gate, o = torch.randn(T, H, generator=g) * 3, torch.randn(T, H * 6, generator=g)
    out = dev(torch.zeros(T, H * 6))
    eng.ops.head_post(dev(o), out, dv=6, gate=dev(gate), gate_per_head=True)
    assert (host(eng, out).view(T, H, 6) - o.double().view(T, H, 6) * torch.sigmoid(gate.double())[:, :, None]).abs().max() < 1e-5


@pytest.mark.parametrize("window,p0,n", [(40, 0, 300), (150, 70, 260), (128, 5, 256), (0, 30, 170), (0, 0, 260)])
def test_latent_prompt_on_the_tensor_cores(window, p0, n):
    """a long portion (serving mode) through the two tensor-core products against the row kernel on the same rows: the
    weights of the value product keep more than bf16's mantissa"""
    eng = _eng(False)
    from mlx_vlm_b200.models.decoder_blocks import LatentAttention
    g = torch.Generator().manual_seed(window + n)
    m = LatentAttention(0, lat(heads=3, kv_rank=64, window=window), 32, gated="head", split_weights=True)
    assert (m.rot_dim, m.row_dim, m.n_gate) == (0, 64, 3)
    T = p0 + n
    pool = _Pool(slots=2, capacity=T + 5, row=64, dtype=torch.bfloat16)
    pool.buf[0, 1, :T] = dev(torch.randn(T, 64, generator=g)).to(torch.bfloat16)
    qa = dev(bf(0.3 * torch.randn(n, 3 * 64, generator=g)))
    ctx = _ctx(eng, pool, [(0, n, 1, p0)])
    a, b = dev(torch.zeros(n, 3 * 64)), dev(torch.zeros(n, 3 * 64))
    with eng.ops.on_stream():
        m._attend_prompt(eng.ops, qa, pool.buf[0][1], ctx.pos, a, p0, n)
        eng.ops.latent_attention(qa, pool.buf[0], ctx.slot, ctx.pos, b, 3, 64, m.scale, n_split=1, window=window)
    assert eng.ops.tc_enabled
    assert (host(eng, a) - host(eng, b)).abs().max() < 2e-3


@pytest.mark.parametrize("taps", [1, 2, 4])
def test_convolution_and_silu_in_portions_and_slots(taps):
    eng = _eng()
    ops = eng.ops
    g = torch.Generator().manual_seed(taps)
    C, n = 37, 23
    c = bf(torch.randn(C, taps, generator=g))
    ha, hb = torch.randn(n, C, generator=g), torch.randn(9, C, generator=g)
    want_a, want_b = O.conv_silu(ha.double(), c.double()), O.conv_silu(hb.double(), c.double())
    pool = _Pool(slots=3, state=(taps - 1) * C + 5)
    st = pool.state[:, 2:2 + (taps - 1) * C]
    got_a, at = [], 0
    for k, cut in enumerate([5, 1, 1, 9, 2, 5]):
        segs, rows = [(0, cut, 2, at)], [ha[at:at + cut]]
        if k == 1:                    # b joins for one step, whole, in slot 0
            segs.append((cut, 9, 0, 0))
            rows.append(hb)
        ctx = _ctx(eng, pool, segs) if (cut > 1 or k == 1) else _decode_ctx(eng, pool, [2], [at])
        y = host(eng, ops.short_conv(dev(torch.cat(rows)), dev(c, torch.bfloat16), st, ctx, act=True))
        got_a.append(y[:cut])
        if k == 1:
            assert (y[cut:] - want_b).abs().max() < 1e-5
        at += cut
    assert (torch.cat(got_a) - want_a).abs().max() < 1e-5
    y = host(eng, ops.short_conv(dev(hb), dev(c, torch.bfloat16), st, _ctx(eng, pool, [(0, 9, 2, 0)]), act=True))
    assert (y - want_b).abs().max() < 1e-5            # slot 2 again, from position 0: what a left there is not read


DELTA_SIZES = [(3, 1, 8, 5), (4, 2, 12, 16), (2, 2, 20, 33), (6, 3, 40, 24), (1, 1, 64, 70), (2, 1, 100, 40), (2, 2, 128, 9),
               (1, 1, 200, 36), (5, 5, 4, 130), (64, 64, 16, 150), (8, 8, 16, 100)]


@pytest.mark.parametrize("H,G,d,dv", DELTA_SIZES)
@pytest.mark.parametrize("cuts", [[17, 1, 1, 2, 25], [46], [31, 1, 9, 5]])
def test_delta_walk_in_portions_and_slots(H, G, d, dv, cuts):
    """the state with a decay per key channel: long portions (walked in chunks, the last one ragged), short ones and single
    tokens (walked token by token), a second sequence beside the first, a slot used again; channels that keep everything,
    channels that forget within a token, and keys that repeat (so that the correction of the delta rule is large)"""
    eng = _eng()
    ops = eng.ops
    from mlx_vlm_b200.models.decoder_blocks import state_floats
    g = torch.Generator().manual_seed(H * 100 + d + len(cuts))
    A_log = bf(torch.randn(H, generator=g))
    dtb = bf(-2.0 + 3.0 * torch.randn(H * d, generator=g))

    def rand(T):
        k = torch.randn(T, G * d, generator=g)
        for t in range(3, T, 3):
            k[t] = k[t - 1] * 1.5 + 0.1 * k[t]
        return [torch.randn(T, G * d, generator=g), k, torch.randn(T, H * dv, generator=g), 2.0 * torch.randn(T, H * d, generator=g),
                2.0 * torch.randn(T, H, generator=g)]

    def ref(q, k, v, x, b):
        T, rep = q.shape[0], H // G
        q, k = (t.double().view(T, G, d) for t in (q, k))
        q, k = O.unit(q) * 0.3, O.unit(k)
        return O.delta_walk(q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1), v.double().view(T, H, dv),
                            O.channel_decay(x.double(), A_log.double(), dtb.double(), H), torch.sigmoid(b.double())).reshape(T, H * dv)

    n = sum(cuts)
    a, b = rand(n), rand(29)
    want_a, want_b = ref(*a), ref(*b)
    tol = lambda w: 3e-5 * max(1.0, w.abs().max().item())
    sf = state_floats(H, d, dv)
    pool = _Pool(slots=3, state=sf + 4)
    st = pool.state[:, 4:4 + sf]

    def run(ctx, parts):
        q, k, v, x, be = (dev(torch.cat(p)) for p in parts)
        o = dev(torch.zeros(q.shape[0], H * dv))
        ops.linear_state(q, k, v, o, st, ctx, H=H, rep=H // G, dim=d, vdim=dv, unit_eps=1e-6, q_scale=0.3, A_log=dev(A_log, torch.bfloat16),
                         dt_bias=dev(dtb, torch.bfloat16), b=be, delta=True, decay_logits=x)
        return host(eng, o)

    got, at = [], 0
    for kk, cut in enumerate(cuts):
        part = [[t[at:at + cut]] for t in a]
        if kk == len(cuts) - 1:       # b joins for one step, whole, in another slot, before a's rows
            y = run(_ctx(eng, pool, [(0, 29, 0, 0), (29, cut, 2, at)]), [[t] + p for p, t in zip(part, b)])
            assert (y[:29] - want_b).abs().max() < tol(want_b)
            y = y[29:]
        elif cut == 1:
            y = run(_decode_ctx(eng, pool, [2], [at]), part)
        else:
            y = run(_ctx(eng, pool, [(0, cut, 2, at)]), part)
        got.append(y)
        at += cut
    assert (torch.cat(got) - want_a).abs().max() < tol(want_a)
    y = run(_ctx(eng, pool, [(0, 29, 2, 0)]), [[t] for t in b])          # slot 2 again, from position 0
    assert (y - want_b).abs().max() < tol(want_b)
    # many single tokens in one step (more rows than the token-by-token kernel takes): every slot goes on by itself
    if H <= 4:
        many = [rand(2) for _ in range(20)]
        pool2 = _Pool(slots=20, state=sf)
        st = pool2.state
        for t in range(2):
            y = run(_decode_ctx(eng, pool2, list(range(20)), [t] * 20), [[m[i][t:t + 1] for m in many] for i in range(5)])
            want = torch.cat([ref(*m)[t:t + 1] for m in many])
            assert (y - want).abs().max() < tol(want)


def test_state_forgets_by_channel():
    """one channel that keeps (decay one to fp32) and one that forgets at once: only the first can answer a far query"""
    eng = _eng()
    ops = eng.ops
    from mlx_vlm_b200.models.decoder_blocks import state_floats
    d, dv, T = 2, 3, 60
    dtb = torch.tensor([-60.0, 30.0])
    k, v = torch.zeros(T, d), torch.zeros(T, dv)
    k[5, 0] = k[6, 1] = 1.0
    v[5], v[6] = torch.tensor([1.0, 2.0, 3.0]), torch.tensor([4.0, 5.0, 6.0])
    q = torch.ones(T, d)
    pool = _Pool(slots=1, state=state_floats(1, d, dv))
    o = dev(torch.zeros(T, dv))
    ops.linear_state(dev(q), dev(k), dev(v), o, pool.state, _ctx(eng, pool, [(0, T, 0, 0)]), H=1, rep=1, dim=d, vdim=dv,
                     unit_eps=1e-6, q_scale=1.0, A_log=dev(torch.zeros(1), torch.bfloat16), dt_bias=dev(dtb, torch.bfloat16),
                     b=dev(torch.full((T, 1), 40.0)), delta=True, decay_logits=dev(torch.zeros(T, d)))
    y = host(eng, o) * math.sqrt(2.0)
    assert (y[6] - torch.tensor([5.0, 7.0, 9.0])).abs().max() < 1e-4
    assert (y[T - 1] - torch.tensor([1.0, 2.0, 3.0])).abs().max() < 1e-4 and y[:5].abs().max() == 0


def test_relu_gated_unit():
    eng, eng16 = _eng(), _eng(False)
    g = torch.Generator().manual_seed(2)
    a, b = torch.randn(40, 56, generator=g) * 3, torch.randn(40, 56, generator=g) * 5
    want = torch.relu(a.double()) * b.double()
    for n in (5, 40):
        out = dev(torch.zeros(n, 56))
        eng.ops.glu_clamp(dev(a[:n]), dev(b[:n]), float("inf"), 1.0, out, up_offset=0.0, relu=True)
        assert (host(eng, out) - want[:n]).abs().max() < 1e-5
    yb = host(eng16, eng16.ops.glu_clamp_bf16(dev(a), dev(b), float("inf"), 1.0, up_offset=0.0, relu=True))
    assert ((yb[:, :56] - want).abs() <= want.abs() / 256).all() and yb[:, 56:].abs().max() == 0


# ------------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt_and_every_layer(dtype):
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
                def wrapped(c, xx, f=f):
                    f(c, xx)
                    seen.append(host(eng, xx))
                L.forward = wrapped
            lm.step([toks], [lm.make_cache()])
        finally:
            for L, f in zip(model.layers, real):
                L.forward = f
        assert len(seen) == len(layers_ref) == 5
        for got, want in zip(seen, layers_ref):
            assert (got - want).abs().max() < 3e-5 * max(1.0, want.abs().max().item())


def test_first_tokens():
    cfg = config()
    model, W = build(cfg)
    for n in (1, 2, 3, 4):
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


@pytest.mark.parametrize("cuts", [[2] * 35, [3, 64, 3], [31, 1, 32, 6], [12, 1, 13, 14, 30], [69, 1], [11, 11, 22, 26], [8, 16, 24, 22]])
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
    assert cc[0]._row == 1 and cc[0].offset == 0
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
    got = host(eng, lm.step([[5]], [cc]))                # c's rows and state survived the move
    assert rel(got, O.forward(cfg, W, c + [5])[-1:]) < TOL["float32"]
    eng.kv_copy_row(pool, 3, pool, 1, cc[0].offset)      # a slot copied to another row (the scheduler's compaction)
    moved = lm.make_cache_row(pool, 3)
    for m in moved:
        m.offset = cc[0].offset
    got = host(eng, lm.step([[9]], [moved]))
    assert rel(got, O.forward(cfg, W, c + [5, 9])[-1:]) < TOL["float32"]


def test_long_prompt_paths_of_the_serving_mode():
    """prompts of 128 tokens and more take the tensor-core products (projections, per-head products, attention in chunks,
    the low-rank projections); a long portion after a cached prefix; a batch whose short member stays on the row kernels"""
    cfg = config([layer("latent_attention", lat(heads=2, dim=64, vdim=16, kv_rank=64, q_rank=24, window=150), 48),
                  layer("channel_delta", delta(heads=4, kv_heads=2, dim=16, vdim=16, conv=4)),
                  layer("attention", att(heads=4, kv_heads=2, dim=24, dims=16, window=40), 40),
                  layer("latent_attention", lat(heads=4, dim=64, vdim=8, kv_rank=64, q_rank=40, window=0, kv_from=0), None),
                  layer("attention", att(heads=2, kv_heads=1, dim=16, dims=16, window=0, scaling=None), 40)], width=64)
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


def test_long_decoding():
    cfg = config()
    model, W = build(cfg)
    toks = tokens(330, cfg["vocab"], 5)
    got = run_alone(model, toks, [20] + [1] * 310)
    assert rel(got, O.forward(cfg, W, toks)) < TOL["float32"]


OTHER = {
    "recurrent layers first, no feed-forward on the attention": config(
        [layer("channel_delta", delta(heads=3, kv_heads=3, dim=24, vdim=8, conv=5), 20), layer("channel_delta", delta(heads=1, kv_heads=1, dim=6, vdim=36)),
         layer("attention", att(heads=2, kv_heads=2, dim=14, dims=14, scaling=None), None)], alpha=0.8),
    "one head, one tap, windows of one, factors of one": config(
        [layer("attention", att(heads=1, kv_heads=1, dim=4, dims=2, window=1, scaling=(1.0, 1.0, 2.0, 16), scale=1.0)),
         layer("channel_delta", delta(heads=1, kv_heads=1, dim=1, vdim=1, conv=1), 8),
         layer("latent_attention", lat(heads=1, dim=1, vdim=1, kv_rank=8, q_rank=4, window=1, scale=1.0), 1)], width=40, vocab=37, alpha=1.0),
    "two lenders, borrowers with wider and narrower windows, no rotation": config(
        [layer("latent_attention", lat(window=5)), layer("attention", att(heads=8, kv_heads=4, dim=10, dims=0, window=64), None),
         layer("latent_attention", lat(heads=2, dim=30, vdim=6, kv_rank=40, window=33), 16),
         layer("latent_attention", lat(heads=7, dim=6, vdim=4, kv_from=0, window=50), None),
         layer("latent_attention", lat(heads=4, dim=9, vdim=11, kv_rank=40, kv_from=2, window=2), 24),
         layer("latent_attention", lat(heads=1, kv_from=0, window=0), None)], width=48, alpha=2.5),
    "equal ranks and sizes, wide heads, an odd vocabulary": config(
        [layer("channel_delta", delta(heads=2, kv_heads=1, dim=72, vdim=72, conv=4, a_rank=16, g_rank=16)),
         layer("attention", att(heads=3, kv_heads=1, dim=72, dims=40, window=64))], width=72, vocab=257),
    "nothing cached": config([layer("channel_delta", delta(heads=3, kv_heads=1, dim=11, vdim=13, conv=6), 25),
                              layer("channel_delta", delta(heads=2, kv_heads=2, dim=33, vdim=10, conv=2), None)], width=52, vocab=77),
    "no state": config([layer("attention", att(heads=5, kv_heads=5, dim=18, dims=6, window=23), 28),
                        layer("latent_attention", lat(heads=6, dim=14, vdim=18, kv_rank=36, window=29), None)], width=60, vocab=89),
    "many heads, odd sizes": config(
        [layer("channel_delta", delta(heads=12, kv_heads=4, dim=5, vdim=7, a_rank=3, g_rank=5)),
         layer("latent_attention", lat(heads=11, dim=5, vdim=3, kv_rank=17, q_rank=9, window=8), 33)], width=45, vocab=61),
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
    from mlx_vlm_b200.sample_utils import make_sampler
    got = [t for t, _ in generate_step(np.asarray([prompt]), model, None, None, max_tokens=6,
                                       sampler=make_sampler(temp=0.0), logit_bias={0: 0.0})]
    same_until_tie(got, want[:6], margins, "generate_step with a sampler")


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
    """bin/trace_run on a checkpoint folder: the registry picks the class from `architecture`, the ranks come from the
    checkpoint's shapes, requests are prefilled together, decoded together, one ends and a later one takes its slot;
    both number formats"""
    import json
    import os
    import subprocess
    import sys
    from safetensors.torch import save_file
    cfg = config()
    W = O.random_weights(cfg, 11, a_rank=5, g_rank=7)
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
