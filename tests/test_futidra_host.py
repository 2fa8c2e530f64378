"""Host-side parts of the Futidra integration (no GPU): configuration, registry, the packed layout of its blocks against
the checkpoint names, cache rows (own, borrowed) and state spans of the layers, the frequency table, the algebra of the
chunked delta walk, and sanity properties of the plain restatement the GPU tests compare with."""
import math

import pytest
import torch

from oracle import futidra as O


def att(**kw):
    m = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 6, "scale": 0.3, "mask": {"size": 5},
         "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 4.0, "original": 16, "low": 1.0, "high": 8.0}}}
    m.update(kw)
    return m


def lat(**kw):
    m = {"heads": 3, "dim": 4, "vdim": 5, "kv_rank": 7, "q_rank": 6, "scale": 0.5, "mask": {"size": 3}}
    m.update(kw)
    return m


def delta(**kw):
    m = {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 9, "conv": 3}
    m.update(kw)
    return m


def config():
    return {"architecture": "Futidra", "vocab": 29, "width": 20, "norm": {"eps": 1e-4}, "postln_alpha": 1.25,
            "layers": [{"type": "channel_delta", "mixer": delta(), "mlp": {"kind": "dense", "ff": 12}},
                       {"type": "latent_attention", "mixer": lat(), "mlp": None},
                       {"type": "attention", "mixer": att(), "mlp": {"kind": "dense", "ff": 8}},
                       {"type": "latent_attention", "mixer": lat(kv_from=1, heads=2, mask={"size": 9}), "mlp": None},
                       {"type": "channel_delta", "mixer": delta(heads=2, dim=9, a_rank=4, g_rank=4, conv=1), "mlp": None}]}


def test_config_and_registry():
    from mlx_vlm_b200.models.futidra import ModelConfig
    from mlx_vlm_b200.utils import get_model_and_args
    c = ModelConfig.from_dict(config())
    assert (c.vocab, c.width, c.norm_eps, c.postln_alpha, c.num_hidden_layers) == (29, 20, 1e-4, 1.25, 5)
    assert ModelConfig.from_dict(c.to_dict()).to_dict() == c.to_dict()
    arch, name = get_model_and_args(config())
    assert name == "futidra" and hasattr(arch, "Model")
    with pytest.raises(ValueError):
        ModelConfig.from_dict({"vocab": 3})
    with pytest.raises(ValueError):
        ModelConfig.from_dict({"vocab": 3, "width": 2, "layers": [{"mixer": {}}]})


def test_model_layout_matches_the_checkpoint_names():
    from mlx_vlm_b200.models.decoder_blocks import NormedSumLayer, state_floats
    from mlx_vlm_b200.models.futidra import Model, ModelConfig
    cfg = config()
    m = Model(ModelConfig.from_dict(cfg), device="cpu")       # no engine is made until something runs
    m._ranks_from(O.random_weights(cfg))                      # the ranks that a checkpoint's shapes give
    assert m.checkpoint_tensors() == O.tensor_shapes(cfg)
    L0, L1, L2, L3, L4 = m.layers
    names = dict(m.manifest())
    # everything that reads the mixer's input is one stacked product; a recurrent layer's is padded to whole vectors
    assert names["l0.mix.in"] == ((2 * 20 + 36 + 8 + 6 + 4 + 7) // 8 * 8, 20) and names["l0.mix.conv"] == (76, 3)
    assert names["l1.mix.down"] == (6 + 7 + 3, 20) and names["l3.mix.down"] == (6 + 2, 20)
    assert names["l2.mix.qkv"] == (4 * 6 + 2 * 6, 20) and names["l2.mix.q.norm"] == (6,)
    assert "l3.mix.dkv.norm" not in names and "l1.norm2" not in names and names["l2.norm2.b"] == (20,) and "head" not in names
    # the second low-rank projections are packed together only when rank and size agree
    assert names["l0.mix.a2"] == (40, 8) and names["l0.mix.g2"] == (36, 6) and names["l4.mix.ag2"] == (2, 18, 4)
    # cache rows: the borrowing layer reads its source's; rows are whole 16-byte vectors
    assert m.n_cache_layers == 2 and m.row_dim == 24
    assert (L1.mixer.cache_index, L2.mixer.cache_index, L3.mixer.cache_index) == (0, 1, 0)
    assert (L1.kv_dim, L2.kv_dim, L3.kv_dim, L0.kv_dim) == (7, 24, 7, 0)
    s0, s4 = 2 * 76 + state_floats(4, 10, 9), state_floats(2, 9, 9)
    assert (L0.state_floats, L4.state_floats, L4.mixer.state_off, m.state_floats) == (s0, s4, s0, s0 + s4)
    assert (L2.mixer.window, L2.mixer.sink, L2.mixer.head_norm, L2.mixer.pairs, L2.mixer.v_from_k, L2.mixer.rot_scaling) == \
        (5, "unit", True, True, True, ("wavelength", 4.0, 16.0, 1.0, 8.0))
    assert (L1.mixer.window, L1.mixer.rot_dim, L1.mixer.gate_per_head, L1.mixer.split_weights, L3.mixer.window) == (3, 0, True, True, 9)
    assert L0.ff.relu and L0.alpha == 1.25
    for bad in ({"type": "other", "mixer": {}}, {"type": "attention", "mixer": att(heads=3), "mlp": None},
                {"type": "attention", "mixer": att(vdim=5), "mlp": None},
                {"type": "attention", "mixer": att(rot={"base": 10.0, "dims": 8}), "mlp": None},
                {"type": "channel_delta", "mixer": delta(heads=3), "mlp": None},
                {"type": "latent_attention", "mixer": lat(), "mlp": {"kind": "other"}}):
        with pytest.raises(ValueError):
            NormedSumLayer(0, bad, 20)
    for src in (4, 2, 0, 3):                                  # not before it, not a latent, not a latent, itself
        bad = config()
        bad["layers"][3]["mixer"]["kv_from"] = src
        with pytest.raises(ValueError):
            Model(ModelConfig.from_dict(bad), device="cpu")
    bad = config()
    bad["layers"][3]["mixer"]["kv_rank"] = 8
    with pytest.raises(ValueError):
        Model(ModelConfig.from_dict(bad), device="cpu")


def test_packing_stacks_the_projections():
    from mlx_vlm_b200.models.decoder_blocks import NormedSumLayer
    cfg = config()
    W = O.random_weights(cfg, 2)
    ck = {k: v.bfloat16() for k, v in W.items()}
    L = NormedSumLayer(0, cfg["layers"][0], 20)
    L.mixer.set_rank("a", 8)
    L.mixer.set_rank("g", 6)
    store = {n: torch.ones(s, dtype=torch.bfloat16) for n, s in L.manifest("l0.")}
    L.pack("l0.", ck, store.__getitem__)
    p = "l0.mix."
    want = torch.cat([W[p + n] for n in ("q", "k", "v", "a1", "g1", "b")])
    assert torch.equal(store[p + "in"].float()[:want.shape[0]], want) and store[p + "in"][want.shape[0]:].abs().max() == 0
    assert torch.equal(store[p + "conv"].float(), torch.cat([W[p + n + ".conv"] for n in "qkv"]))
    assert torch.equal(store["l0.mlp.gu"].float(), torch.cat([W["l0.mlp.gate"], W["l0.mlp.up"]])) and L.w["norm1.b"] is store["l0.norm1.b"]
    L = NormedSumLayer(4, cfg["layers"][4], 20)
    store = {n: torch.zeros(s, dtype=torch.bfloat16) for n, s in L.manifest("l4.")}
    L.pack("l4.", {k: v.bfloat16() for k, v in O.random_weights(cfg, 2).items()}, store.__getitem__)
    assert torch.equal(store["l4.mix.ag2"].float(), torch.stack([W["l4.mix.a2"], W["l4.mix.g2"]]))
    L = NormedSumLayer(3, cfg["layers"][3], 20)
    store = {n: torch.zeros(s, dtype=torch.bfloat16) for n, s in L.manifest("l3.")}
    L.pack("l3.", ck, store.__getitem__)
    assert torch.equal(store["l3.mix.down"].float(), torch.cat([W["l3.mix.dq"], W["l3.mix.g"]]))
    assert torch.equal(store["l3.mix.ukT"].float(), W["l3.mix.uk"].view(2, 4, 7).transpose(1, 2))


def test_borrowed_rows_are_shared_views():
    from mlx_vlm_b200.models.cache import RunCache, StatePool
    pool = StatePool(2, 24, 8, "cpu", batch=2, capacity=16, dtype=torch.float32)
    own, borrowed = RunCache(pool, 1, kv_layer=0, kv_dim=7), RunCache(pool, 1, kv_layer=0, kv_dim=7, shared=True)
    pool.buf[0, 1, 3] = 2.0
    assert torch.equal(own.keys, borrowed.keys) and borrowed.keys[0, 3, 0] == 2.0
    assert borrowed.nbytes == 0 and own.nbytes == own.keys.numel() * 4


# ---- the plain restatement itself ---------------------------------------------------------------------------
def test_restatement_frequencies_and_rotation():
    sc = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}
    plain, f = O.frequencies(1000.0, 32, None), O.frequencies(1000.0, 32, sc)
    for a, b in zip(plain, f):
        turns = 512 * a / (2 * math.pi)
        if turns > 4.0:
            assert b == a
        elif turns < 1.0:
            assert b == a / 8.0
        else:
            assert a / 8.0 <= b <= a
    assert f[0] == plain[0] and f[-1] == plain[-1] / 8.0 and f == sorted(f, reverse=True)
    v = torch.randn(3, 2, 6, dtype=torch.float64)
    pos = torch.tensor([0, 1, 9])
    r = O.rotate_pairs(v, pos, {"base": 10.0, "dims": 4})
    assert torch.equal(r[0], v[0]) and torch.equal(r[..., 4:], v[..., 4:])
    assert torch.allclose(r[1, :, 0], v[1, :, 0] * math.cos(1) - v[1, :, 1] * math.sin(1))
    assert torch.allclose(r[..., 2:4].norm(dim=-1), v[..., 2:4].norm(dim=-1))


def test_restatement_windows_sink_and_state():
    a = [3, 1, 4, 1, 5, 9, 2, 6]
    b = [7] + a[1:]                                            # another first token
    base = {"architecture": "Futidra", "vocab": 17, "width": 12, "norm": {"eps": 1e-5}, "postln_alpha": 1.5}

    def run(layer, toks):
        cfg = {**base, "layers": [layer]}
        return O.forward(cfg, O.random_weights(cfg, 1), toks)

    for layer in ({"type": "attention", "mixer": att(heads=2, kv_heads=1, mask={"size": 3}), "mlp": None},
                  {"type": "latent_attention", "mixer": lat(), "mlp": {"kind": "dense", "ff": 8}}):
        za, zb = run(layer, a), run(layer, b)
        assert (za[:3] - zb[:3]).abs().max() > 1e-6 and (za[3:] - zb[3:]).abs().max() < 1e-12     # the window holds 3 tokens
        assert (run(layer, a[:5]) - za[:5]).abs().max() < 1e-12                                    # causal
    za, zb = (run({"type": "channel_delta", "mixer": delta(), "mlp": None}, t) for t in (a, b))
    assert (za[-1] - zb[-1]).abs().max() > 1e-9                # the state remembers the first token
    s = torch.tensor([[[-30.0, 0.0], [-30.0, -30.0]]])
    w = O.softmax(s, O.visible(2, 0), True)
    assert w.abs().max() < 1e-6                                # nothing but the added one
    assert torch.allclose(O.softmax(s, O.visible(2, 0), False).sum(-1), torch.ones(1, 2))


def test_delta_rule_in_chunks_is_the_token_by_token_rule():
    """the chunk form the kernels compute — decays multiplied between two tokens of a chunk, never divided by — against the
    token-by-token restatement, with decays down to zero"""
    g = torch.Generator().manual_seed(0)
    T, d, dv, C = 24, 6, 5, 8
    q, k = (O.unit(torch.randn(T, 1, d, generator=g, dtype=torch.float64)) for _ in range(2))
    k[5] = k[4]
    v = torch.randn(T, 1, dv, generator=g, dtype=torch.float64)
    dec = torch.rand(T, 1, d, generator=g, dtype=torch.float64)
    dec[3, 0, 1] = dec[9, 0, 2] = 0.0
    beta = torch.rand(T, 1, generator=g, dtype=torch.float64)
    want = O.delta_walk(q, k, v, dec, beta)[:, 0]
    S, got = torch.zeros(d, dv, dtype=torch.float64), []
    for c in range(0, T, C):
        kc, qc, vc, gc, bc = (t[c:c + C, 0] for t in (k, q, v, dec, beta[..., None]))
        through = lambda s, t: gc[s + 1:t + 1].prod(0)                      # decays after token s up to token t
        G = [gc[:t + 1].prod(0) for t in range(C)]
        A = torch.tensor([[float((kc[t] * kc[s] * through(s, t)).sum()) if s < t else 0.0 for s in range(C)] for t in range(C)], dtype=torch.float64)
        B = torch.tensor([[float((qc[t] * kc[s] * through(s, t)).sum()) if s <= t else 0.0 for s in range(C)] for t in range(C)], dtype=torch.float64)
        Tm = torch.linalg.inv(torch.eye(C, dtype=torch.float64) + torch.diag(bc[:, 0]) @ A) @ torch.diag(bc[:, 0])
        w = vc - torch.stack([G[t] * kc[t] for t in range(C)]) @ S
        got.append(torch.stack([G[t] * qc[t] for t in range(C)]) @ S + B @ Tm @ w)
        S = G[-1][:, None] * S + torch.stack([through(t, C - 1) * kc[t] for t in range(C)]).T @ (Tm @ w)
    assert (torch.cat(got) - want).abs().max() < 1e-12
