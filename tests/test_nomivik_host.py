"""Host-side parts of the Nomivik integration (no GPU): configuration, registry, order of the layer runs, the packed layout
of its blocks against the checkpoint names, cache rows and state spans of every run, the algebra of the matrix memory taken
many tokens at a time, and sanity properties of the plain restatement the GPU tests compare with."""
import pytest
import torch

from oracle import nomivik as O


def left(**kw):
    return dict({"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "scale": 0.3, "softcap": 9.0, "mask": {"size": 5},
                 "rot": {"base": 100.0, "dims": 4}}, **kw)


def right(**kw):
    return dict({"heads": 3, "dim": 4, "vdim": 7, "gate_cap": 11.0}, **kw)


def pair(mlp=12, **kw):
    return {"type": "parallel", "mixer": {"left": left(**kw), "right": right()}, "mlp": {"kind": "dense", "ff": mlp} if mlp else None}


def lru(mlp=None, **kw):
    return {"type": "rglru", "mixer": dict({"width": 10, "blocks": 2, "conv": 3}, **kw), "mlp": {"kind": "dense", "ff": mlp} if mlp else None}


def config(**kw):
    return dict({"architecture": "Nomivik", "vocab": 29, "width": 20, "norm": {"eps": 1e-4}, "layers": [lru(), pair(), lru(8, conv=1), pair(None)],
                 "loop": {"start": 1, "stop": 3, "times": 2}, "token_side": {"dim": 3},
                 "embedding": {"bigram": {"buckets": 17, "mul_prev": 5, "mul_cur": 3}}}, **kw)


def test_config_and_registry():
    from mlx_vlm_b200.models.nomivik import ModelConfig
    from mlx_vlm_b200.utils import get_model_and_args
    c = ModelConfig.from_dict(config())
    assert (c.vocab, c.width, c.norm_eps, c.side_dim, c.num_hidden_layers) == (29, 20, 1e-4, 3, 6)
    assert c.layer_runs() == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)] == O.layer_runs(4, config()["loop"])
    assert ModelConfig.from_dict(c.to_dict()).to_dict() == c.to_dict()
    bare = ModelConfig.from_dict({"vocab": 3, "width": 2, "layers": [lru()]})
    assert bare.loop is None and bare.bigram is None and bare.side_dim == 0 and bare.layer_runs() == [(0, False)]
    arch, name = get_model_and_args(config())
    assert name == "nomivik" and hasattr(arch, "Model")
    for bad in ({"vocab": 3}, config(layers=[{"mixer": {}}]), config(loop={"start": 2, "stop": 5, "times": 1}),
                config(loop={"start": 2, "stop": 2, "times": 1}), config(embedding={"bigram": {"buckets": 0, "mul_prev": 1, "mul_cur": 1}})):
        with pytest.raises(ValueError):
            ModelConfig.from_dict(bad)


def test_model_layout_matches_the_checkpoint_names():
    from mlx_vlm_b200.models.decoder_blocks import PreNormLayer
    from mlx_vlm_b200.models.nomivik import Model, ModelConfig
    cfg = config()
    m = Model(ModelConfig.from_dict(cfg), device="cpu")       # no engine is made until something runs
    assert m.checkpoint_tensors() == O.tensor_shapes(cfg)
    names = dict(m.manifest())
    # everything that reads the mixer's input is one stacked product, padded to whole vectors, with one bias
    n_in = (24 + 12 + 10) + (12 + 12 + 21 + 21 + 3 + 3)
    assert names["l1.mix.in"] == ((n_in + 7) // 8 * 8, 20) and names["l1.mix.in.b"] == ((n_in + 7) // 8 * 8,)
    assert names["l0.mix.yx"] == (20, 20) and names["l0.mix.gates"] == (2, 10, 5) and names["l2.mix.conv"] == (10, 1)
    assert "l0.norm2" not in names and names["l2.norm2"] == (20,) and "head" not in names and names["side.embed"] == (29, 12)
    # every run has its own rows and its own span of the state, behind the last token
    assert (m.n_cache_layers, m.row_dim) == (3, 24)
    par_state, rec, rec1 = (3 * (4 * 8 + 1) + 3) // 4 * 4, (2 * 10 + 10 + 3) // 4 * 4, (10 + 3) // 4 * 4
    offs = [4]
    for n in (rec, par_state, rec1, par_state, rec1, par_state):
        offs.append(offs[-1] + n)
    assert [r.state_base for r in m.runs] + [m.state_floats] == offs
    assert [r.kv_base for r in m.runs] == [0, 0, 1, 1, 2, 2] and [r.opens_pass for r in m.runs] == [False] * 3 + [True, False, False]
    L = m.layers[1].mixer
    assert (L.left.window, L.left.sink, L.left.unit_norm, L.left.softcap, L.left.bias, L.left.pairs, L.right.cap, L.factor) == \
        (5, "unit", True, 9.0, True, False, 11.0, 0.5)
    assert m.layers[0].mixer.decay == 8.0
    for bad in ({"type": "other", "mixer": {}}, pair(kv_heads=3), pair(rot={"base": 10.0, "dims": 8}), lru(blocks=3),
                dict(lru(), mlp={"kind": "other"})):
        with pytest.raises(ValueError):
            PreNormLayer(0, bad, 20)


def test_packing_stacks_the_projections():
    from mlx_vlm_b200.models.decoder_blocks import PreNormLayer
    cfg = config()
    W = O.random_weights(cfg, 2)
    ck = {k: v.bfloat16() for k, v in W.items()}
    L = PreNormLayer(1, cfg["layers"][1], 20, side_dim=3)
    store = {n: torch.ones(s, dtype=torch.bfloat16) for n, s in L.manifest("l1.")}
    L.pack("l1.", ck, store.__getitem__)
    p = "l1.mix."
    want = torch.cat([W[p + n] for n in ("left.q", "left.k", "left.v", "right.q", "right.k", "right.v", "right.g", "right.i", "right.f")])
    n = want.shape[0]
    assert torch.equal(store[p + "in"].float()[:n], want) and store[p + "in"][n:].abs().sum() == 0
    b = store[p + "in.b"].float()
    assert torch.equal(b[:46], torch.cat([W[p + "left." + s + ".b"] for s in "qkv"])) and b[46:n - 6].abs().max() == 0
    assert torch.equal(b[n - 6:n], torch.cat([W[p + "right.i.b"], W[p + "right.f.b"]])) and b[n:].abs().sum() == 0
    assert L.mixer.right.w["norm"] is store[p + "right.norm"] and L.side.w["gate"] is store["l1.side.gate"]
    L = PreNormLayer(0, cfg["layers"][0], 20, side_dim=3)
    store = {n: torch.ones(s, dtype=torch.bfloat16) for n, s in L.manifest("l0.")}
    L.pack("l0.", ck, store.__getitem__)
    assert torch.equal(store["l0.mix.gates"].float(), torch.cat([W["l0.mix.ra"], W["l0.mix.ri"]], 1))
    assert torch.equal(store["l0.mix.yx"].float(), torch.cat([W["l0.mix.y"], W["l0.mix.x"]]))
    assert torch.equal(store["l0.mix.ri.b"].float(), W["l0.mix.ri.b"].reshape(-1))


def test_runs_of_one_layer_keep_apart():
    from mlx_vlm_b200.models.cache import StatePool
    from mlx_vlm_b200.models.nomivik import Model, ModelConfig
    m = Model(ModelConfig.from_dict(config()), device="cpu")
    pool = StatePool(m.n_cache_layers, m.row_dim, m.state_floats, "cpu", batch=2, capacity=8, dtype=torch.float32)
    caches = m.language_model.make_cache_row(pool, 1)
    assert len(caches) == 6 and not any(c.is_trimmable() for c in caches)
    for i, c in enumerate(caches):
        c.recurrent.fill_(float(i + 1))
    assert [float(c.recurrent.mean()) for c in caches] == [1.0, 2.0, 3.0, 4.0, 5.0, 6.0] and pool.state[0].abs().max() == 0
    assert pool.state[1, :4].abs().max() == 0                  # the last token's number is nobody's
    assert caches[1].keys.data_ptr() != caches[3].keys.data_ptr() and caches[0].keys is None


# ---- the plain restatement itself ---------------------------------------------------------------------------
def test_restatement_bigram_rotation_and_cap():
    assert O.bigram_rows([4, 9, 9], 5, 3, 17) == [17, (20 + 27) % 17, (45 + 27) % 17]
    v = torch.randn(3, 2, 6, dtype=torch.float64)
    r = O.rotate_half(v, torch.tensor([0, 1, 9]), {"base": 10.0, "dims": 4})
    assert torch.equal(r[0], v[0]) and torch.equal(r[..., 4:], v[..., 4:])
    c, s = torch.cos(torch.tensor(1.0, dtype=torch.float64)), torch.sin(torch.tensor(1.0, dtype=torch.float64))
    assert torch.allclose(r[1, :, 0], v[1, :, 0] * c - v[1, :, 2] * s) and torch.allclose(r[1, :, 2], v[1, :, 2] * c + v[1, :, 0] * s)
    assert torch.allclose(O.rms(r, 1e-3), O.rotate_half(O.rms(v, 1e-3), torch.tensor([0, 1, 9]), {"base": 10.0, "dims": 4}))
    x = torch.tensor([-900.0, 0.0, 0.01, 900.0], dtype=torch.float64)
    assert torch.allclose(O.capped(x, 3.0), torch.tensor([-3.0, 0.0, 0.01, 3.0], dtype=torch.float64), atol=1e-6) and O.capped(x, None) is x
    w = O.softmax_with_one(torch.tensor([[[-40.0, 0.0], [-40.0, -40.0]]]), O.visible(2, 0))
    assert w.max() < 1e-6                                      # nothing but the added one


def test_restatement_window_state_and_loop():
    a = [3, 1, 4, 1, 5, 9, 2, 6]
    b = [7] + a[1:]                                            # another first token

    def run(layers, toks, **kw):
        cfg = config(layers=layers, loop=None, **kw)
        W = O.random_weights(cfg, 1)
        if kw.get("mute"):
            for n in W:
                if n.endswith("right.out"):
                    W[n].zero_()
        return O.forward(cfg, W, toks)

    za, zb = (run([pair(mask={"size": 3})], t, mute=True) for t in (a, b))
    # the window holds 3 tokens, and the bigram carries the first token one position further
    assert (za[2] - zb[2]).abs().max() > 1e-6 and (za[4:] - zb[4:]).abs().max() < 1e-12
    for layer in (pair(), lru()):
        za, zb = run([layer], a), run([layer], b)
        assert (za[-1] - zb[-1]).abs().max() > 1e-9            # the state remembers the first token
        assert (run([layer], a[:5]) - za[:5]).abs().max() < 1e-12                                      # causal
    one, two = (config(layers=[lru()], loop={"start": 0, "stop": 1, "times": k}) for k in (1, 2))
    W = O.random_weights(one, 3)
    assert (O.forward(one, W, a) - O.forward(dict(one, loop=None), W, a)).abs().max() == 0
    assert (O.forward(two, W, a) - O.forward(one, W, a)).abs().max() > 1e-3


def test_matrix_memory_in_chunks_is_the_token_by_token_rule():
    """the chunk form the kernels compute (sums of log forget gates within a chunk, the running maximum before it) against the
    token-by-token restatement, with input gates that overtake the maximum and forget gates that drop everything"""
    g = torch.Generator().manual_seed(0)
    T, d, dv, C = 24, 6, 5, 8
    q, k = (torch.randn(T, 1, d, generator=g, dtype=torch.float64) for _ in range(2))
    v = torch.randn(T, 1, dv, generator=g, dtype=torch.float64)
    i = 3.0 * torch.randn(T, 1, generator=g, dtype=torch.float64)
    f = torch.nn.functional.logsigmoid(2.0 + 3.0 * torch.randn(T, 1, generator=g, dtype=torch.float64))
    i[11], f[5] = 12.0, -50.0
    want = O.memory_walk(q, k, v, i, f)[:, 0]
    S, m, got = torch.zeros(d, dv + 1, dtype=torch.float64), 0.0, []
    for c in range(0, T, C):
        qc, kc, ic = q[c:c + C, 0], k[c:c + C, 0], i[c:c + C, 0]
        vc = torch.cat([v[c:c + C, 0], torch.ones(C, 1, dtype=torch.float64)], 1)        # the normaliser is one more column
        F = torch.cumsum(f[c:c + C, 0], 0)
        mt = torch.stack([torch.maximum(F[t] + m, (F[t] - F[:t + 1] + ic[:t + 1]).max()) for t in range(C)])
        w = torch.exp((F[:, None] - F[None, :] + ic[None, :] - mt[:, None]).masked_fill(~O.visible(C, 0), float("-inf")))
        assert w.max() <= 1.0
        o = torch.exp(F + m - mt)[:, None] * (qc @ S) + (w * (qc @ kc.T)) @ vc
        got.append(o[:, :dv] / (torch.maximum(o[:, dv].abs(), torch.exp(-mt)) + 1e-6)[:, None])
        S = torch.exp(F[-1] + m - mt[-1]) * S + (kc * w[-1][:, None]).T @ vc
        m = mt[-1]
    assert (torch.cat(got) - want).abs().max() < 1e-11
