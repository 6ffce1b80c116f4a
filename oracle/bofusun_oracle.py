"""Float64 restatement of the Bofusun design, one function per mechanism, for the tests.  Shares no code with the package.

A model is a dict `cfg` in the layout of the design's config.json and a dict `w` of tensors under the checkpoint's names.
Notation: T tokens of ONE sequence, rows are time steps; every function takes and returns float64 tensors.

    N(x; w) = x / sqrt(mean(x^2) + eps) * (1 + w)
    e = N(E[id]; w_e);  x = e
    layers start .. stop-1 run `times` times:  ahead of pass t  x <- x + e (t > 0);  x <- x + step_t
    layer:  x <- x + N(mixer(N(x)));   with a feed-forward  x <- x + N(ff(N(x)))
    logits = W_head N(x; w_f)
"""
import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def causal_conv(u, w, bias=None, history=None):
    """y[t, c] = sum_j w[c, j] u[t - K + 1 + j, c] (+ bias[c]); rows ahead of the sequence are zeros, or `history` ([K-1, C], oldest
    first) when the sequence is continued."""
    T, C = u.shape
    K = w.shape[1]
    full = torch.cat([torch.zeros((K - 1, C), dtype=F64) if history is None else history, u], 0)
    y = torch.zeros((T, C), dtype=F64)
    for j in range(K):
        y += full[j:j + T] * w[:, j]
    return y if bias is None else y + bias


def rotate_half(x, pos, dims, base):
    """x [T, heads, dim]: entries i and i + dims/2 (i < dims/2) turn by pos * base^(-2i/dims); the rest pass."""
    if dims == 0:
        return x
    half = dims // 2
    f = torch.tensor(base, dtype=F64) ** (-2.0 * torch.arange(half, dtype=F64) / dims)
    ang = pos.to(F64)[:, None] * f[None, :]
    c, s = ang.cos()[:, None, :], ang.sin()[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], -1)


def retention(q, k, v, decay, S=None):
    """Per head: S = decay S + k v^T; o = S^T q.  q, k [T, H, d]; v [T, H, dv]; decay [H].  Returns o and the last S [H, d, dv]."""
    T, H, d = q.shape
    S = torch.zeros((H, d, v.shape[2]), dtype=F64) if S is None else S.clone()
    o = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for t in range(T):
        S = S * decay[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def retention_mixer(h, w, p, m, pos, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    r = m.get("rot") or {}
    q = rotate_half((h @ w[p + "q"].T).view(T, H, d), pos, int(r.get("dims", 0)), float(r.get("base", 10000.0)))
    k = rotate_half((h @ w[p + "k"].T).view(T, H, d), pos, int(r.get("dims", 0)), float(r.get("base", 10000.0))) * d ** -0.5
    v = (h @ w[p + "v"].T).view(T, H, dv)
    o, _ = retention(q, k, v, torch.tensor(m["decay"], dtype=F64))
    return (unit_rms(o, eps).reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def bucket(n, rows, far):
    """Row of the distance table for distance n >= 0: exact below rows / 2, then logarithmic up to `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def biased_attention(q, k, v, scale, cap, rel, far, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; score = cap tanh(scale q.k / cap) + rel[bucket(i - j), h] over the last `window` keys."""
    T, H, d = q.shape
    G = k.shape[1]
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    see = (dist >= 0) & (dist < window)
    idx = torch.tensor([bucket(n, rel.shape[0], far) for n in range(T)])[dist.clamp(min=0)]
    out = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = cap * torch.tanh((q[:, h] @ k[:, g].T) * scale / cap) + rel[:, h][idx]
        out[:, h] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g]
    return out


def attention_mixer(h, w, p, m):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    u = {n: causal_conv(h @ w[p + n].T + w[p + n + ".b"], w[p + n + ".conv"]) for n in "qkv"}
    o = biased_attention(u["q"].view(T, H, d), u["k"].view(T, G, d), u["v"].view(T, G, dv), float(m["scale"]), float(m["softcap"]),
                         w[p + "rel"], float(m["bias_max"]), int(m["mask"]["size"]))
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def selective_scan(x, dt, A, B, C, D, S=None):
    """Per channel c and state n: S = exp(dt_c A[c, n]) S + dt_c x_c B_n; y_c = sum_n S C_n + D_c x_c.  Returns y and the last S."""
    T, c = x.shape
    S = torch.zeros_like(A) if S is None else S.clone()
    y = torch.zeros((T, c), dtype=F64)
    for t in range(T):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def mamba_mixer(h, w, p, m):
    inner, R, N = m["inner"], m["dt_rank"], m["state"]
    xz = h @ w[p + "in"].T
    x = silu(causal_conv(xz[:, :inner], w[p + "conv"], w[p + "conv.b"]))
    f = x @ w[p + "x"].T
    dt = softplus(f[:, :R] @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), f[:, R:R + N], f[:, R + N:], w[p + "D"])
    return (y * silu(xz[:, inner:])) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    a = attention_mixer(h, w, p + "left.", m["left"])
    b = mamba_mixer(h, w, p + "right.", m["right"])
    return 0.5 * (unit_rms(a, eps) * w[p + "left.out"] + unit_rms(b, eps) * w[p + "right.out"])


def dense_ff(h, w, p):
    return torch.clamp(h @ w[p + "up"].T + w[p + "up.b"], min=0.0) ** 2 @ w[p + "down"].T + w[p + "down.b"]


def passes(cfg):
    """[(layer, pass)] in the order they run; pass is None outside the loop."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    return [(i, None) for i in range(a)] + [(i, t) for t in range(int(loop["times"])) for i in range(a, b)] + [(i, None) for i in range(b, n)]


def forward(cfg: dict, w: Dict[str, torch.Tensor], ids: List[int], streams_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence run as a whole; `streams_out` receives the residual after every layer run."""
    w = {k: v.to(F64) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    pos = torch.arange(len(ids))
    e = norm(w["embed"][torch.tensor(ids)], w["embed.norm"], eps)
    x = e
    for i, t in passes(cfg):
        if t is not None and i == int(cfg["loop"]["start"]):
            x = (x + e if t > 0 else x) + w["loop.step"][t]
        L, p = cfg["layers"][i], f"l{i}."
        h = norm(x, w[p + "norm1"], eps)
        if L["type"] == "retention":
            y = retention_mixer(h, w, p + "mix.", L["mixer"], pos, eps)
        elif L["type"] == "parallel":
            y = parallel_mixer(h, w, p + "mix.", L["mixer"], eps)
        else:
            raise ValueError(L["type"])
        x = x + norm(y, w[p + "norm1b"], eps)
        if L.get("mlp"):
            x = x + norm(dense_ff(norm(x, w[p + "norm2"], eps), w, p + "mlp."), w[p + "norm2b"], eps)
        if streams_out is not None:
            streams_out.append(x)
    return norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, w, prompt: List[int], n_new: int) -> List[int]:
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(forward(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt):]
