"""Small Bofusun configurations with random weights for the tests: a config.json-shaped dict and bf16-exact weights under the
checkpoint's tensor names.  The engine helpers (replay, rel_rms, write_checkpoint, make_engine) are those of stack_util."""
import torch

from conftest import pkg
from stack_util import bf16_exact


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def retention(heads=3, dim=20, vdim=12, rot_dims=16, base=3000.0, decay=None, mlp=None):
    decay = decay or [1.0 - 2.0 ** -(2 + 0.8 * h) for h in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": rot_dims}}, "mlp": mlp}


def parallel(heads=4, kv_heads=2, dim=20, vdim=12, window=17, conv=2, scale=0.3, softcap=4.0, bias_max=40, rows=10, inner=28, state=5, dt_rank=3,
             conv2=3, mlp=None):
    """`rows`: rows of the distance table (a tensor's size, not part of the configuration)."""
    return {"type": "parallel", "rows": rows, "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "conv": conv, "scale": scale,
                               "softcap": softcap, "bias_max": bias_max},
                      "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv2}}}


def make_cfg(width=56, vocab=110, layers=None, eps=1e-5, loop=(1, 3, 2)):
    """loop: (start, stop, times) or None."""
    if layers is None:
        layers = [parallel(mlp=dense()), retention(), parallel(heads=3, kv_heads=1, dim=16, vdim=24, window=40, conv=4, inner=44, state=18, dt_rank=9, conv2=2),
                  retention(heads=2, dim=36, vdim=40, rot_dims=20, mlp=dense(24))]
    return {"architecture": "Bofusun", "norm": {"eps": eps}, "vocab": vocab, "width": width, "layers": layers,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))}


def make_weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(o, i, s=None):
        return bf16_exact(torch.randn(o, i, generator=g) * (s if s is not None else i ** -0.5))

    def vec(k, mean=0.0, jitter=0.1):
        return bf16_exact(mean + jitter * torch.randn(k, generator=g))

    w = {"embed": mat(V, W, 0.7), "embed.norm": vec(W), "final.norm": vec(W), "head": mat(V, W)}
    if cfg.get("loop"):
        w["loop.step"] = mat(cfg["loop"]["times"], W, 0.4)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        for q in ("1", "1b") + (("2", "2b") if L["mlp"] else ()):
            w[p + "norm" + q] = vec(W)
        if L["type"] == "retention":
            H, d, e = m["heads"], m["dim"], m["vdim"]
            w[p + "mix.q"], w[p + "mix.k"], w[p + "mix.v"], w[p + "mix.g"] = mat(H * d, W), mat(H * d, W), mat(H * e, W), mat(H * e, W)
            w[p + "mix.o"] = mat(W, H * e)
        else:
            a, b = m["left"], m["right"]
            H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "mix.left."
            for n, ch in (("q", H * d), ("k", G * d), ("v", G * e)):
                w[q + n], w[q + n + ".b"], w[q + n + ".conv"] = mat(ch, W), vec(ch, 0.0, 0.5), mat(ch, a["conv"], 0.7)
            w[q + "rel"], w[q + "g"], w[q + "o"], w[q + "out"] = mat(L["rows"], H, 1.0), mat(H, W), mat(W, H * e), vec(W, 1.0, 0.2)
            q, I, N, R = p + "mix.right.", b["inner"], b["state"], b["dt_rank"]
            w[q + "in"], w[q + "conv"], w[q + "conv.b"] = mat(2 * I, W), mat(I, b["conv"], 0.6), vec(I, 0.0, 0.3)
            w[q + "x"], w[q + "dt"], w[q + "dt.b"] = mat(R + 2 * N, I), mat(I, R), vec(I, -1.0, 1.0)
            w[q + "A_log"], w[q + "D"], w[q + "o"], w[q + "out"] = mat(I, N, 0.8), vec(I, 1.0, 0.5), mat(W, I), vec(W, 1.0, 0.2)
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            w[p + "mlp.up"], w[p + "mlp.up.b"], w[p + "mlp.down"], w[p + "mlp.down.b"] = mat(ff, W), vec(ff, 0.0, 0.3), mat(W, ff), vec(W, 0.0, 0.3)
    return w


def product_config(cfg):
    return pkg("config").BofusunConfig.from_dict(cfg, name="test")


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
