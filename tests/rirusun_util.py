"""Small Rirusun configurations with random weights for the tests: a config.json-shaped dict and bf16-exact weights under the
checkpoint's tensor names.  The engine helpers (replay, rel_rms, write_checkpoint, make_engine) are those of stack_util."""
import torch

from conftest import pkg
from stack_util import bf16_exact

YARN = {"factor": 4.0, "original": 48, "fast": 6.0, "slow": 0.5}


def moe(experts=8, top=3, ff=24, groups=(4, 2), shared=20):
    """groups: (count, keep) or None; shared: the shared expert's size or None."""
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    f = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def mlstm(heads=3, dim=20, vdim=12, cap=6.0, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def latent(heads=3, dim=20, rot_dim=12, vdim=14, kv_rank=28, scale=0.3, base=700.0, scaling=YARN, mlp=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(scaling)
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                              "scale": scale, "rot": rot}}


def parallel(heads=4, kv_heads=2, dim=20, vdim=12, window=17, keep=3, scale=0.3, bias_max=40, rows=10, width=36, blocks=3, conv=3, mix=(0.7, 1.3), mlp=None):
    """`rows`: rows of the distance table (a tensor's size, not part of the configuration)."""
    return {"type": "parallel", "rows": rows, "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "keep_first": keep}, "scale": scale,
                               "bias_max": bias_max},
                      "right": {"width": width, "blocks": blocks, "conv": conv}, "left_scale": mix[0], "right_scale": mix[1]}}


def make_cfg(width=56, vocab=110, layers=None, eps=1e-5, loop=(1, 3, 2), scale=3.0):
    """loop: (start, stop, times) or None."""
    if layers is None:
        layers = [latent(mlp=moe()), parallel(mlp=moe(experts=6, top=2, groups=(3, 2), ff=40, shared=None)),
                  mlstm(mlp=moe(experts=4, top=2, groups=None, ff=16)),
                  parallel(heads=3, kv_heads=1, dim=16, vdim=24, window=30, keep=5, width=40, blocks=2, conv=4, bias_max=25, rows=8, mix=(1.0, 0.5))]
    return {"architecture": "Rirusun", "embedding": {"scale": scale}, "norm": {"eps": eps}, "vocab": vocab, "width": width, "layers": layers,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))}


def make_weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(o, i, s=None):
        return bf16_exact(torch.randn(o, i, generator=g) * (s if s is not None else i ** -0.5))

    def vec(k, mean=0.0, jitter=0.1):
        return bf16_exact(mean + jitter * torch.randn(k, generator=g))

    w = {"embed": mat(V, W, 0.3), "head": mat(V, W)}

    def norm(name):
        w[name], w[name + ".b"], w[name + ".alpha"] = vec(W, 1.0, 0.2), vec(W, 0.0, 0.2), bf16_exact(torch.tensor(0.6))

    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        norm(p + "norm1")
        q = p + "mix."
        if L["type"] == "mlstm":
            H, d, e = m["heads"], m["dim"], m["vdim"]
            w[q + "q"], w[q + "k"], w[q + "v"], w[q + "g"], w[q + "o"] = mat(H * d, W), mat(H * d, W), mat(H * e, W), mat(H * e, W), mat(W, H * e)
            w[q + "i"], w[q + "f"], w[q + "norm"] = mat(H, W), mat(H, W), vec(H * e, 1.0, 0.2)
            w[q + "i.b"], w[q + "f.b"] = vec(H, 0.0, 0.5), vec(H, 3.0, 1.0)
        elif L["type"] == "latent_attention":
            H, d, r, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w[q + "q"], w[q + "dkv"], w[q + "dkv.norm"] = mat(H * (d + r), W, 1.5 * W ** -0.5), mat(R + r, W, 1.5 * W ** -0.5), vec(R, 1.0, 0.2)
            w[q + "uk"], w[q + "uv"], w[q + "o"] = mat(H * d, R), mat(H * e, R), mat(W, H * e)
        else:
            a, b = m["left"], m["right"]
            H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            l, r = q + "left.", q + "right."
            w[l + "q"], w[l + "k"], w[l + "v"], w[l + "o"] = mat(H * d, W), mat(G * d, W), mat(G * e, W), mat(W, H * e)
            w[l + "q.norm"], w[l + "k.norm"], w[l + "rel"], w[l + "sink"] = vec(H * d, 1.0, 0.3), vec(G * d, 1.0, 0.3), mat(L["rows"], H, 1.0), vec(H, 0.5, 1.0)
            n, k = b["width"], b["blocks"]
            for x in "xy":
                w[r + x], w[r + x + ".b"] = mat(n, W), vec(n, 0.0, 0.3)
            w[r + "conv"], w[r + "conv.b"] = mat(n, b["conv"], 0.6), vec(n, 0.0, 0.3)
            for x in ("ra", "ri"):
                w[r + x], w[r + x + ".b"] = mat(n, n // k).view(k, n // k, n // k), vec(n, 0.0, 0.5).view(k, n // k)
            w[r + "lam"], w[r + "o"] = vec(n, -4.0, 2.0), mat(W, n)
        f = L["mlp"]
        if f:
            E, ff, p = f["router"]["experts"], f["expert"]["ff"], p + "mlp."
            w[p + "router"] = mat(E, W, 3.0 * W ** -0.5)     # spread-out scores: few near-ties
            w[p + "correction"] = vec(E, -0.6, 0.3)          # choice scores of either sign
            for j in range(E):
                w[f"{p}e{j}.up"], w[f"{p}e{j}.down"] = mat(ff, W), mat(W, ff)
            if f.get("shared"):
                s = f["shared"]["ff"]
                w[p + "shared.up"], w[p + "shared.down"], w[p + "shared.sg"] = mat(s, W), mat(W, s), mat(1, W)
    return w


def product_config(cfg):
    return pkg("config").RirusunConfig.from_dict(cfg, name="test")


def make_runner(cfg, w, dtype="float32", **kw):
    kw.setdefault("max_tokens", 512)
    kw.setdefault("max_model_len", 1024)
    kw.setdefault("block_size", 16)
    kw.setdefault("n_blocks", 80)
    kw.setdefault("max_logit_rows", 512)
    kw.setdefault("n_state_slots", 5)
    r = pkg("runner").make_runner(product_config(cfg), dtype=dtype, **kw)
    r.load_weights({k: v.clone() for k, v in w.items()})
    return r
