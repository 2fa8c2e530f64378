"""ORACLE — TEST INFRASTRUCTURE ONLY. Not imported by the product path.

Plain, slow restatement of the Futidra decoder, one function per mechanism, written from the design's equations with
torch on the CPU.  It shares no code with mlx_vlm_b200/: no cache, no state objects, no batching; every call walks
the whole sequence.

Notation: x (T, W) residual stream, a = `postln_alpha`.  A layer norms the SUM, the sublayers read x itself:
    x <- N1(a x + mixer(x));   x <- N2(a x + ff(x)),      N(y) = (y - mean) / sqrt(mean((y - mean)^2) + eps) * w + b.
Mixers:
  'attention'         grouped heads whose values are the projected keys (before norm and rotation); RMS norm per head on
                      q and k with one weight for all heads; rotary in pairs (2i, 2i + 1) on the first dims numbers of a
                      head, frequencies rescaled by wavelength; sliding window; one added to the softmax's denominator;
  'latent_attention'  queries through a normed latent, keys and values expanded from one normed latent row per token (the
                      layer's own, or an earlier layer's), no positions, sliding window, plain softmax, a sigmoid gate
                      per head;
  'channel_delta'     delta rule with a decay per head and key channel on a (dim, vdim) state per head; short convolutions
                      and silu on q, k, v; unit-length q, k; per-head RMS norm and a low-rank sigmoid gate on the output.
Feed-forward: W_down (relu(W_gate x) * (W_up x)).  Output: N with 'final.norm', then the embedding table.

Weights: dict name -> tensor with the checkpoint's names ('embed', 'l<i>.norm1', 'l<i>.norm1.b', 'l<i>.mix.q', ...).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------------------------------------ pieces
def layer_norm(y: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = y - y.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms(y: torch.Tensor, eps: float) -> torch.Tensor:
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


def post_norm(x: torch.Tensor, y: torch.Tensor, alpha: float, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    return layer_norm(alpha * x + y, w, b, eps)


def frequencies(base: float, dims: int, scaling: Optional[dict]) -> List[float]:
    """f_i = base^(-2i/dims); with a scaling, by the wavelength l = 2 pi / f: short waves keep f, long ones take f / factor,
    between them the two are blended linearly in original / l"""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > original / low:
                f = f / factor
            elif wave >= original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate_pairs(v: torch.Tensor, pos: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """v (T, heads, D): of the first `dims` numbers of a head, (2i, 2i + 1) is a pair turned by pos * f_i"""
    dims = int((rot or {}).get("dims", 0))
    if dims < 2:
        return v.clone()
    f = torch.tensor(frequencies(float(rot["base"]), dims, rot.get("scaling")), dtype=torch.float64)
    a = pos.to(torch.float64)[:, None] * f[None, :]
    cos, sin = torch.cos(a).to(v.dtype)[:, None, :], torch.sin(a).to(v.dtype)[:, None, :]
    out = v.clone()
    even, odd = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = even * cos - odd * sin
    out[..., 1:dims:2] = odd * cos + even * sin
    return out


def visible(T: int, size: int) -> torch.Tensor:
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (dist >= 0) & (dist < size) if size else dist >= 0


def window(c: dict) -> int:
    return int((c.get("mask") or {}).get("size", 0))


def softmax(s: torch.Tensor, seen: torch.Tensor, plus_one: bool) -> torch.Tensor:
    """s (H, T, T) scores, seen (T, T) bool -> weights; plus_one: the denominator is 1 + sum exp(s)"""
    s = s.masked_fill(~seen[None], float("-inf"))
    m = s.max(-1, keepdim=True).values
    if plus_one:
        m = m.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + (torch.exp(-m) if plus_one else 0.0))


def attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, c: dict, pos: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q, k = (h @ w[p + "q"].T).view(T, H, d), (h @ w[p + "k"].T).view(T, G, d)
    v = k
    q = rotate_pairs(rms(q, eps) * w[p + "q.norm"], pos, c.get("rot"))
    k = rotate_pairs(rms(k, eps) * w[p + "k.norm"], pos, c.get("rot"))
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    a = softmax(torch.einsum("thd,shd->hts", q, k) * float(c["scale"]), visible(T, window(c)), True)
    return torch.einsum("hts,shd->thd", a, v).reshape(T, H * d) @ w[p + "o"].T


def latent_rows(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    return rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]


def latent_attention(h: torch.Tensor, c_rows: torch.Tensor, w: Dict[str, torch.Tensor], p: str, c: dict,
                     eps: float) -> torch.Tensor:
    """c_rows (T, kv_rank): the latent rows the layer reads (its own or another layer's)"""
    T, H, d, dv = h.shape[0], c["heads"], c["dim"], c["vdim"]
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).view(T, H, d)
    k, v = (c_rows @ w[p + "uk"].T).view(T, H, d), (c_rows @ w[p + "uv"].T).view(T, H, dv)
    a = softmax(torch.einsum("thd,shd->hts", q, k) * float(c["scale"]), visible(T, window(c)), False)
    o = torch.einsum("hts,shd->thd", a, v) * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def conv_silu(u: torch.Tensor, c: torch.Tensor) -> torch.Tensor:
    """u (T, C), c (C, taps): y_t = silu(sum_j c[:, j] u_(t - taps + 1 + j)), zeros before the sequence"""
    T, taps = u.shape[0], c.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += c[:, j] * u[:T - back]
    return y * torch.sigmoid(y)


def unit(y: torch.Tensor) -> torch.Tensor:
    return y / torch.sqrt((y * y).sum(-1, keepdim=True) + 1e-6)


def delta_walk(q, k, v, g, beta) -> torch.Tensor:
    """q, k, g (T, H, dim), v (T, H, vdim), beta (T, H): token by token  S <- diag(g) S;  u = beta (v - S^T k);
    S <- S + k u^T;  o = S^T q"""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hij,hi->hj", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hij,hi->hj", S, q[t])
    return o


def channel_decay(x: torch.Tensor, A_log: torch.Tensor, dt_bias: torch.Tensor, H: int) -> torch.Tensor:
    """x (T, H dim) projected -> g (T, H, dim) = exp(-exp(A_log_h) softplus(x + dt_bias))"""
    z = torch.nn.functional.softplus(x + dt_bias, threshold=50.0)
    return torch.exp(-torch.exp(A_log)[:, None] * z.view(x.shape[0], H, -1))


def channel_delta(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, c: dict, eps: float) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (conv_silu(h @ w[p + n].T, w[p + n + ".conv"]) for n in "qkv")
    q, k = unit(q.view(T, G, d)) * d ** -0.5, unit(k.view(T, G, d))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    g = channel_decay((h @ w[p + "a1"].T) @ w[p + "a2"].T, w[p + "A_log"], w[p + "dt_bias"], H)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    o = rms(delta_walk(q, k, v.view(T, H, dv), g, beta), eps) * w[p + "norm"]
    o = o.reshape(T, H * dv) * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return o @ w[p + "o"].T


def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (torch.relu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, return_layers: bool = False, dtype=torch.float64):
    """tokens: one sequence from position 0.  -> logits (T, vocab) (and the residual stream after every layer)"""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in w.items()}
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    tok = torch.as_tensor(tokens, dtype=torch.long)
    pos = torch.arange(tok.shape[0])
    x = w["embed"][tok]
    latents: Dict[int, torch.Tensor] = {}
    after: List[torch.Tensor] = []
    for i, L in enumerate(cfg["layers"]):
        p, c, kind = f"l{i}.", L["mixer"], L["type"]
        if kind == "attention":
            y = attention(x, w, p + "mix.", c, pos, eps)
        elif kind == "latent_attention":
            src = c.get("kv_from")
            if src is None:
                src = i
                latents[i] = latent_rows(x, w, p + "mix.", eps)
            y = latent_attention(x, latents[src], w, p + "mix.", c, eps)
        elif kind == "channel_delta":
            y = channel_delta(x, w, p + "mix.", c, eps)
        else:
            raise ValueError(kind)
        x = post_norm(x, y, alpha, w[p + "norm1"], w[p + "norm1.b"], eps)
        if L.get("mlp") is not None:
            x = post_norm(x, dense_ff(x, w, p + "mlp."), alpha, w[p + "norm2"], w[p + "norm2.b"], eps)
        after.append(x)
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
    return (logits, after) if return_layers else logits


# ------------------------------------------------------------------------------------------------ test weights
def tensor_shapes(cfg: dict, a_rank: int = 8, g_rank: int = 6) -> Dict[str, tuple]:
    """checkpoint name -> shape of every tensor of a configuration"""
    W, V = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": (V, W), "final.norm": (W,), "final.norm.b": (W,)}
    for i, L in enumerate(cfg["layers"]):
        p, c = f"l{i}.", L["mixer"]
        m = p + "mix."
        out.update({p + "norm1": (W,), p + "norm1.b": (W,)})
        H, d, dv = c["heads"], c["dim"], c["vdim"]
        out[m + "o"] = (W, H * dv)
        if L["type"] == "attention":
            G = c["kv_heads"]
            out.update({m + "q": (H * d, W), m + "k": (G * d, W), m + "q.norm": (d,), m + "k.norm": (d,)})
        elif L["type"] == "latent_attention":
            r, rq = c["kv_rank"], c["q_rank"]
            out.update({m + "dq": (rq, W), m + "dq.norm": (rq,), m + "uq": (H * d, rq), m + "uk": (H * d, r),
                        m + "uv": (H * dv, r), m + "g": (H, W)})
            if c.get("kv_from") is None:
                out.update({m + "dkv": (r, W), m + "dkv.norm": (r,)})
        else:
            n, nv, taps = c["kv_heads"] * d, H * dv, c["conv"]
            ra, rg = int(c.get("a_rank", a_rank)), int(c.get("g_rank", g_rank))
            out.update({m + "q": (n, W), m + "k": (n, W), m + "v": (nv, W), m + "q.conv": (n, taps), m + "k.conv": (n, taps),
                        m + "v.conv": (nv, taps), m + "b": (H, W), m + "A_log": (H,), m + "norm": (dv,), m + "a1": (ra, W),
                        m + "a2": (H * d, ra), m + "dt_bias": (H * d,), m + "g1": (rg, W), m + "g2": (nv, rg)})
        if L.get("mlp") is not None:
            f = L["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "norm2.b": (W,), p + "mlp.gate": (f, W), p + "mlp.up": (f, W),
                        p + "mlp.down": (W, f)})
    return out


def random_weights(cfg: dict, seed: int = 0, gain: float = 1.0, a_rank: int = 8, g_rank: int = 6) -> Dict[str, torch.Tensor]:
    """bf16-valued random weights (stored as float32): matrices N(0, gain^2 / fan-in), norm weights around one, decays from
    a few tokens to hundreds, convolutions that mix their taps"""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, a_rank, g_rank).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif last == "b" and len(shape) == 1:
            t = 0.2 * torch.randn(shape, generator=g)
        elif last == "A_log":
            t = 0.5 * torch.randn(shape, generator=g)
        elif last == "dt_bias":
            t = -3.5 + 1.5 * torch.randn(shape, generator=g)
        elif last == "conv":
            t = 0.5 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * gain / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out
