"""ORACLE — TEST INFRASTRUCTURE ONLY. Not imported by the product path.

Plain, slow restatement of the Nomivik decoder, one function per mechanism, written from the design's equations with
torch on the CPU.  It shares no code with mlx_vlm_b200/: no cache, no state objects, no batching; every call walks
the whole sequence.

Notation: x (T, W) residual stream, N(y) = y / sqrt(mean(y^2) + eps) * w.
    x = embed[t_j] + bigram[(a t_(j-1) + b t_j) mod B]     (the first token: row B)
    layer:  x += mixer(N1(x));   x += ff(N2(x));   x += N_s(P ((gelu(G x)) * s_i[t_j]))   (s_i: layer i's slice of a token table)
    a span of layers runs several times; before every pass after the first the embedding output is added to x.
Mixers:
  'parallel'  two mixers on the same input; half the sum of their outputs, each with a norm over the width:
      left    grouped heads with biases, rotate-half rotary, unit-mean-square q and k, soft-capped scores, a sliding window,
              one added to the softmax's denominator;
      right   a matrix memory per head with exponential input gate, sigmoid-log forget gate and a running maximum;
  'rglru'     a gelu branch times a gated linear recurrence per channel behind a short convolution.
Feed-forward: W_down (silu(W_gate x) * (W_up x)).  Output: N with 'final.norm', then the embedding table.

Weights: dict name -> tensor with the checkpoint's names ('embed', 'bigram', 'l<i>.norm1', 'l<i>.mix.left.q', ...).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------------------------------------ pieces
def rms(y: torch.Tensor, eps: float) -> torch.Tensor:
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


def gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_rows(tokens: List[int], mul_prev: int, mul_cur: int, buckets: int) -> List[int]:
    return [buckets if j == 0 else (int(tokens[j - 1]) * mul_prev + int(t) * mul_cur) % buckets for j, t in enumerate(tokens)]


def embedding(tokens: List[int], w: Dict[str, torch.Tensor], cfg: dict) -> torch.Tensor:
    x = w["embed"][torch.as_tensor(tokens)]
    b = (cfg.get("embedding") or {}).get("bigram")
    if b:
        x = x + w["bigram"][torch.as_tensor(bigram_rows(tokens, b["mul_prev"], b["mul_cur"], b["buckets"]))]
    return x


def layer_runs(n_layers: int, loop: Optional[dict]) -> List[tuple]:
    """[(layer, opens a pass after the first)] in the order the layers run"""
    if not loop:
        return [(i, False) for i in range(n_layers)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, False) for i in range(a)]
    for k in range(times):
        out += [(i, k > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n_layers)]


def rotate_half(v: torch.Tensor, pos: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """v (T, heads, D): number i of the first dims is paired with number i + dims / 2, turned by pos * base^(-2i/dims)"""
    dims = int((rot or {}).get("dims", 0))
    if dims < 2:
        return v.clone()
    half = dims // 2
    f = torch.tensor([float(rot["base"]) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = pos.to(torch.float64)[:, None] * f[None, :]
    cos, sin = torch.cos(a).to(v.dtype)[:, None, :], torch.sin(a).to(v.dtype)[:, None, :]
    out = v.clone()
    lo, hi = v[..., :half], v[..., half:dims]
    out[..., :half] = lo * cos - hi * sin
    out[..., half:dims] = hi * cos + lo * sin
    return out


def visible(T: int, size: int) -> torch.Tensor:
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (dist >= 0) & (dist < size) if size else dist >= 0


def capped(s: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return s if not cap else cap * torch.tanh(s / cap)


def softmax_with_one(s: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
    """s (H, T, T) scores, seen (T, T) bool -> exp(s_j) / (1 + sum exp(s))"""
    s = s.masked_fill(~seen[None], float("-inf"))
    m = s.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-m))


def attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, c: dict, pos: torch.Tensor, eps: float) -> torch.Tensor:
    T, H, d = h.shape[0], c["heads"], c["dim"]
    G, dv = c["kv_heads"], c["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    q, k = rms(rotate_half(q, pos, c.get("rot")), eps), rms(rotate_half(k, pos, c.get("rot")), eps)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    s = capped(torch.einsum("thd,shd->hts", q, k) * float(c["scale"]), c.get("softcap"))
    a = softmax_with_one(s, visible(T, int((c.get("mask") or {}).get("size", 0))))
    return torch.einsum("hts,shd->thd", a, v).reshape(T, H * dv) @ w[p + "o"].T


def memory_walk(q, k, v, i, f) -> torch.Tensor:
    """q, k (T, H, dim), v (T, H, vdim), i, f (T, H) log gates: token by token  m' = max(f + m, i);
    S <- exp(f + m - m') S + exp(i - m') k v^T, n likewise with k alone;  o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)"""
    T, H, d = q.shape
    S, n, m = torch.zeros(H, d, v.shape[-1], dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[t] = torch.einsum("hij,hi->hj", S, q[t]) / den[:, None]
    return o


def matrix_memory(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, c: dict, eps: float) -> torch.Tensor:
    T, H, d, dv, cap = h.shape[0], c["heads"], c["dim"], c["vdim"], float(c["gate_cap"])
    q, k = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5, (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    i = capped(h @ w[p + "i"].T + w[p + "i.b"], cap)
    f = torch.nn.functional.logsigmoid(capped(h @ w[p + "f"].T + w[p + "f.b"], cap))
    o = rms(memory_walk(q, k, v, i, f), eps).reshape(T, H * dv)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w, p, c, pos, eps):
    left = rms(attention(h, w, p + "left.", c["left"], pos, eps), eps) * w[p + "left.out"]
    right = rms(matrix_memory(h, w, p + "right.", c["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (left + right)


def conv(u: torch.Tensor, c: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u (T, C), c (C, taps): y_t = b + sum_j c[:, j] u_(t - taps + 1 + j), zeros before the sequence"""
    T, taps = u.shape[0], c.shape[1]
    y = b[None, :].repeat(T, 1)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] = y[back:] + c[:, j] * u[:T - back]
    return y


def block_linear(u: torch.Tensor, m: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u (T, blocks n), m (blocks, n, n) [out, in], b (blocks, n)"""
    T = u.shape[0]
    return (torch.einsum("tbi,boi->tbo", u.view(T, m.shape[0], -1), m) + b).reshape(T, -1)


def recurrence(u, r, i, lam) -> torch.Tensor:
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u, log a = -8 r softplus(lam)"""
    log_a = -8.0 * r * torch.nn.functional.softplus(lam, threshold=50.0)
    a, z = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    S, out = torch.zeros_like(u[0]), torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + z[t]
        out[t] = S
    return out


def rglru(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    y = gelu(h @ w[p + "y"].T + w[p + "y.b"])
    u = conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(block_linear(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_linear(u, w[p + "ri"], w[p + "ri.b"]))
    return (recurrence(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    g = h @ w[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def token_side(x: torch.Tensor, e: torch.Tensor, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    """e (T, dim): the layer's slice of the tokens' rows"""
    return rms((gelu(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T, eps) * w[p + "side.norm"]


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, return_layers: bool = False, dtype=torch.float64):
    """tokens: one sequence from position 0.  -> logits (T, vocab) (and the residual stream after every layer run)"""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in w.items()}
    eps, side = float(cfg["norm"]["eps"]), cfg.get("token_side")
    tok = [int(t) for t in tokens]
    pos = torch.arange(len(tok))
    x0 = embedding(tok, w, cfg)
    x = x0.clone()
    after: List[torch.Tensor] = []
    for i, opens in layer_runs(len(cfg["layers"]), cfg.get("loop")):
        if opens:
            x = x + x0
        L, p = cfg["layers"][i], f"l{i}."
        h = rms(x, eps) * w[p + "norm1"]
        if L["type"] == "parallel":
            x = x + parallel(h, w, p + "mix.", L["mixer"], pos, eps)
        elif L["type"] == "rglru":
            x = x + rglru(h, w, p + "mix.")
        else:
            raise ValueError(L["type"])
        if L.get("mlp") is not None:
            x = x + dense_ff(rms(x, eps) * w[p + "norm2"], w, p + "mlp.")
        if side:
            n = int(side["dim"])
            x = x + token_side(x, w["side.embed"][tok][:, i * n:(i + 1) * n], w, p, eps)
        after.append(x)
    logits = (rms(x, eps) * w["final.norm"]) @ w["embed"].T
    return (logits, after) if return_layers else logits


# ------------------------------------------------------------------------------------------------ test weights
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """checkpoint name -> shape of every tensor of a configuration"""
    W, V = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": (V, W), "final.norm": (W,)}
    big, side = (cfg.get("embedding") or {}).get("bigram"), cfg.get("token_side")
    if big:
        out["bigram"] = (big["buckets"] + 1, W)
    if side:
        out["side.embed"] = (V, len(cfg["layers"]) * side["dim"])
    for i, L in enumerate(cfg["layers"]):
        p, c = f"l{i}.", L["mixer"]
        m = p + "mix."
        out[p + "norm1"] = (W,)
        if L["type"] == "parallel":
            a, r = c["left"], c["right"]
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                out.update({m + "left." + n: (rows, W), m + "left." + n + ".b": (rows,)})
            out.update({m + "left.o": (W, a["heads"] * a["vdim"]), m + "left.out": (W,), m + "right.out": (W,)})
            H, nv = r["heads"], r["heads"] * r["vdim"]
            out.update({m + "right.q": (H * r["dim"], W), m + "right.k": (H * r["dim"], W), m + "right.v": (nv, W),
                        m + "right.g": (nv, W), m + "right.o": (W, nv), m + "right.norm": (nv,), m + "right.i": (H, W),
                        m + "right.i.b": (H,), m + "right.f": (H, W), m + "right.f.b": (H,)})
        else:
            n, nb = c["width"], c["blocks"]
            out.update({m + "y": (n, W), m + "y.b": (n,), m + "x": (n, W), m + "x.b": (n,), m + "conv": (n, c["conv"]),
                        m + "conv.b": (n,), m + "lam": (n,), m + "o": (W, n)})
            for g in ("ra", "ri"):
                out.update({m + g: (nb, n // nb, n // nb), m + g + ".b": (nb, n // nb)})
        if L.get("mlp") is not None:
            f = L["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.gate": (f, W), p + "mlp.up": (f, W), p + "mlp.down": (W, f)})
        if side:
            out.update({p + "side.gate": (side["dim"], W), p + "side.proj": (W, side["dim"]), p + "side.norm": (W,)})
    return out


def random_weights(cfg: dict, seed: int = 0, gain: float = 1.0) -> Dict[str, torch.Tensor]:
    """bf16-valued random weights (stored as float32): matrices N(0, gain^2 / fan-in), norm weights around one, forget gates
    and decays from a few tokens to hundreds, convolutions that mix their taps"""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm", "out"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif name.endswith("right.f.b"):
            t = 3.0 + 2.0 * torch.randn(shape, generator=g)
        elif last == "b":
            t = 0.3 * torch.randn(shape, generator=g)
        elif last == "lam":
            t = -5.0 + 2.0 * torch.randn(shape, generator=g)
        elif last == "conv":
            t = 0.5 * torch.randn(shape, generator=g)
        elif name in ("embed", "side.embed", "bigram"):
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * gain / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out
