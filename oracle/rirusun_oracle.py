"""Float64 restatement of the Rirusun design, one function per mechanism, for the tests.  Shares no code with the package.

A model is a dict `cfg` in the layout of the design's config.json and a dict `w` of tensors under the checkpoint's names.
Notation: T tokens of ONE sequence, rows are time steps; every function takes and returns float64 tensors.

    D(x; a, w, b) = tanh(a x) w + b                       elementwise, a one number
    x = s E[id];   layers start .. stop-1 run `times` times with the same weights, each pass on its own cache and state
    layer:  h = D(x);  x <- x + mixer(h) + experts(h)     one norm for both
    logits = W_head D(x; final)
"""
import math
from typing import Dict, List, Optional, Tuple

import torch

F64 = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def tanh_norm(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


# ---- latent attention -------------------------------------------------------------------------------------------------------
def rotary_frequencies(base: float, dims: int, scaling: Optional[dict]) -> Tuple[torch.Tensor, float]:
    """(frequency of every pair, factor on cos and sin): with scaling, pairs that make many turns over `original` positions keep
    theirs, pairs that make few are slowed by `factor`, a linear ramp over the pair index between."""
    i = torch.arange(dims // 2, dtype=F64)
    f = float(base) ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0
    at = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(scaling["fast"])), 0), min(math.ceil(at(scaling["slow"])), dims - 1)
    r = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * r + f * (1.0 - r), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_half(x, pos, rot: Optional[dict]):
    """x [T, heads, n]: entries i and i + dims/2 (i < dims/2) turn by pos * f_i; what lies beyond dims passes."""
    dims = int((rot or {}).get("dims") or 0)
    if dims == 0:
        return x
    f, mag = rotary_frequencies(float(rot["base"]), dims, rot.get("scaling"))
    ang = pos.to(F64)[:, None] * f
    c, s = (ang.cos() * mag)[:, None, :], (ang.sin() * mag)[:, None, :]
    a, b = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], -1)


def latent_mixer(h, w, p, m, pos, eps):
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    kv = h @ w[p + "dkv"].T
    c = unit_rms(kv[:, :R], eps) * w[p + "dkv.norm"]
    qr = rotate_half(q[..., d:], pos, m.get("rot"))
    kr = rotate_half(kv[:, None, R:], pos, m.get("rot"))[:, 0]
    k, v = (c @ w[p + "uk"].T).view(T, H, d), (c @ w[p + "uv"].T).view(T, H, dv)
    later = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    out = torch.zeros((T, H, dv), dtype=F64)
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + qr[:, i] @ kr.T) * float(m["scale"])
        out[:, i] = torch.softmax(s.masked_fill(later, -math.inf), -1) @ v[:, i]
    return out.reshape(T, H * dv) @ w[p + "o"].T


# ---- windowed attention with kept first tokens, a distance bias and a sink ---------------------------------------------------
def bucket(n: int, rows: int, far: float) -> int:
    """Row of the distance table for distance n >= 0: exact below rows / 2, then logarithmic up to `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def visible(T: int, window: int, keep: int):
    """[T, T] bool: query i sees key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    return see & ((i - j < window) | (j < keep)) if window > 0 else see


def kept_attention(q, k, v, scale, rel, far, sink, window, keep):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: score = scale q.k + rel[bucket(i - j), h]; exp(sink_h) joins the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    see = visible(T, window, keep)
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    idx = torch.tensor([bucket(n, rel.shape[0], far) for n in range(T)])[dist]
    out = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale + rel[:, h][idx]).masked_fill(~see, -math.inf)
        s = torch.cat([s, sink[h].expand(T, 1)], 1)
        out[:, h] = torch.softmax(s, -1)[:, :T] @ v[:, g]
    return out


def attention_mixer(h, w, p, m, eps):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, d)
    k = (unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, d)
    v = (h @ w[p + "v"].T).view(T, G, dv)
    mask = m.get("mask") or {}
    o = kept_attention(q, k, v, float(m["scale"]), w[p + "rel"], float(m["bias_max"]), w[p + "sink"], int(mask.get("size") or 0),
                       int(mask.get("keep_first") or 0))
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ---- real-gated linear recurrent unit ----------------------------------------------------------------------------------------
def causal_conv(u, w, b):
    """y[t, c] = b[c] + sum_j w[c, j] u[t - K + 1 + j, c], zeros ahead of the sequence."""
    T, K = u.shape[0], w.shape[1]
    full = torch.cat([torch.zeros((K - 1, u.shape[1]), dtype=F64), u], 0)
    return b + sum(full[j:j + T] * w[:, j] for j in range(K))


def block_gate(u, w, b):
    """sigmoid of a block-diagonal product: u [T, C], w [blocks, C/blocks, C/blocks] ([out, in]), b [blocks, C/blocks]."""
    n, s = w.shape[0], w.shape[1]
    return torch.cat([torch.sigmoid(u[:, i * s:(i + 1) * s] @ w[i].T + b[i]) for i in range(n)], 1)


def gated_lru(u, r, i, lam, S=None):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam).  Returns every S_t."""
    S = torch.zeros(u.shape[1], dtype=F64) if S is None else S
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        a = torch.exp(-8.0 * r[t] * softplus(lam))
        S = a * S + torch.sqrt(1.0 - a * a) * i[t] * u[t]
        out[t] = S
    return out


def recurrent_mixer(h, w, p, m):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    S = gated_lru(u, block_gate(u, w[p + "ra"], w[p + "ra.b"]), block_gate(u, w[p + "ri"], w[p + "ri.b"]), w[p + "lam"])
    return (S * y) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    return float(m["left_scale"]) * attention_mixer(h, w, p + "left.", m["left"], eps) \
        + float(m["right_scale"]) * recurrent_mixer(h, w, p + "right.", m["right"])


# ---- matrix memory ------------------------------------------------------------------------------------------------------------
def matrix_memory(q, k, v, log_i, log_f):
    """q, k [T, H, d], v [T, H, dv], gates [T, H]; the running maximum starts at zero.  Returns o [T, H, dv]."""
    T, H, d = q.shape
    S, n, m = torch.zeros((H, d, v.shape[2]), dtype=F64), torch.zeros((H, d), dtype=F64), torch.zeros(H, dtype=F64)
    o = torch.zeros((T, H, v.shape[2]), dtype=F64)
    for t in range(T):
        new = torch.maximum(log_f[t] + m, log_i[t])
        keep, take = torch.exp(log_f[t] + m - new), torch.exp(log_i[t] - new)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[t] = (S * q[t][:, :, None]).sum(1) / den[:, None]
    return o


def memory_mixer(h, w, p, m, eps):
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    T = h.shape[0]
    q, k, v = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5, (h @ w[p + "k"].T).view(T, H, d), (h @ w[p + "v"].T).view(T, H, dv)
    capped = lambda z: cap * torch.tanh(z / cap)
    log_i, log_f = capped(h @ w[p + "i"].T + w[p + "i.b"]), -softplus(-capped(h @ w[p + "f"].T + w[p + "f.b"]))
    o = unit_rms(matrix_memory(q, k, v, log_i, log_f), eps).reshape(T, H * dv)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- routed experts -----------------------------------------------------------------------------------------------------------
def route(z, correction, r: dict):
    """Router logits [T, E] -> (chosen ids [T, top], weights [T, top]): sigmoid scores, the correction joins for the choice only, a
    group counts by the sum of its two best, experts outside the best groups are out, weights sum to one."""
    E, top = r["experts"], r["top"]
    s = torch.sigmoid(z)
    c = s + correction
    g = r.get("groups") or {}
    n, keep = int(g.get("count") or 1), int(g.get("keep") or 1)
    ids, wts = [], []
    for t in range(z.shape[0]):
        parts = c[t].view(n, E // n)
        score = parts.topk(min(2, E // n), -1).values.sum(-1)
        best = set(score.topk(keep).indices.tolist())
        open_ = torch.tensor([e // (E // n) in best for e in range(E)])
        pick = c[t].masked_fill(~open_, -math.inf).topk(top).indices
        ids.append(pick)
        wts.append(s[t][pick] / (s[t][pick].sum() + 1e-20))
    return torch.stack(ids), torch.stack(wts)


def experts(h, w, p, f: dict):
    ids, wts = route(h @ w[p + "router"].T, w[p + "correction"], f["router"])
    one = lambda q, x: gelu_erf(x @ w[q + "up"].T) @ w[q + "down"].T
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(ids.shape[1]):
            y[t] += wts[t, j] * one(f"{p}e{int(ids[t, j])}.", h[t])
    if f.get("shared"):
        y = y + one(p + "shared.", h) * torch.sigmoid(h @ w[p + "shared.sg"].T)
    return y


# ---- the model ----------------------------------------------------------------------------------------------------------------
def passes(cfg) -> List[int]:
    """The layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def forward(cfg: dict, w: Dict[str, torch.Tensor], ids: List[int], streams_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence run as a whole; `streams_out` receives the residual after every layer run."""
    w = {k: v.to(F64) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    pos = torch.arange(len(ids))
    norm = lambda x, n: tanh_norm(x, w[n + ".alpha"], w[n], w[n + ".b"])
    x = w["embed"][torch.tensor(ids)] * float(cfg["embedding"]["scale"])
    for i in passes(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        h = norm(x, p + "norm1")
        if L["type"] == "latent_attention":
            y = latent_mixer(h, w, p + "mix.", L["mixer"], pos, eps)
        elif L["type"] == "parallel":
            y = parallel_mixer(h, w, p + "mix.", L["mixer"], eps)
        elif L["type"] == "mlstm":
            y = memory_mixer(h, w, p + "mix.", L["mixer"], eps)
        else:
            raise ValueError(L["type"])
        if L.get("mlp"):
            y = y + experts(h, w, p + "mlp.", L["mlp"])
        x = x + y
        if streams_out is not None:
            streams_out.append(x)
    return norm(x, "final.norm") @ w["head"].T


def greedy(cfg, w, prompt: List[int], n_new: int) -> List[int]:
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(forward(cfg, w, ids)[-1].argmax()))
    return ids[len(prompt):]
