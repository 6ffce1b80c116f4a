"""Bofusun without a GPU: the registry and every part of the configuration, the unrolled layer list, the weight mapping (fusions,
padded projections, the expanded distance table, norm weights stored around zero), and the oracle's own invariants (causality,
recurrences carried across portions, the window's edges, the buckets of the distance table, what a pass of the loop adds)."""
import math

import pytest
import torch

import bofusun_util as B
import stack_util as U
from conftest import pkg
from oracle import bofusun_oracle as O

F64 = torch.float64


def test_registry_reads_the_layer_list(tmp_path):
    cfg = B.make_cfg()
    path = str(tmp_path / "ckpt")
    U.write_checkpoint(path, cfg, B.make_weights(cfg, 1))
    C = pkg("config")
    pc = C.load_model_config(path)
    assert type(pc).__name__ == "BofusunConfig" and C.is_stack_config(pc) and pc.needs_state
    assert (pc.width, pc.vocab, pc.norm_eps, pc.loop_start, pc.loop_stop, pc.loop_times) == (56, 110, 1e-5, 1, 3, 2)
    assert pc.layer_runs() == [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (3, None)] and pc.n_layers == 6 and len(pc.layers) == 4
    a, s, r = pc.layers[0].mixer, pc.layers[0].side, pc.layers[3].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.conv, a.scale, a.softcap, a.bias_max) == (4, 2, 20, 12, 17, 2, 0.3, 4.0, 40.0)
    assert a.bias and a.head_gate and not a.qk_norm and a.rot is None
    assert (s.inner, s.state, s.dt_rank, s.conv, s.dt_pad, s.proj_rows) == (28, 5, 3, 3, 8, 24)
    assert (r.heads, r.kv_heads, r.dim, r.vdim, r.rot.dims, r.rot.base, len(r.decay)) == (2, 2, 36, 40, 20, 3000.0, 2)
    f = pc.layers[0].mlp
    assert (f.kind, f.ff, f.act, f.gated, f.bias) == ("dense", 40, "relu2", False, True) and pc.layers[1].mlp is None and pc.layers[1].side is None
    assert pc.kv_bytes_per_token() == 2 * (2 * 32 + 2 * 40) and pc.kv_bytes_per_token(True) == 2 * pc.kv_bytes_per_token()


def test_configuration_errors_and_defaults():
    C = pkg("config").BofusunConfig.from_dict
    bad = B.retention()
    bad["mixer"]["decay"] = [0.5]
    for layers, loop in (([{"type": "mlstm", "mixer": {}, "mlp": None}], None), ([bad], None), ([B.retention(rot_dims=22)], None),
                         ([B.retention(rot_dims=7)], None), ([B.parallel(heads=3, kv_heads=2)], None), ([B.retention(mlp={"kind": "moe"})], None),
                         ([B.retention()], (0, 2, 2)), ([B.retention()], (0, 0, 2)), ([B.retention()], (0, 1, 0))):
        with pytest.raises(ValueError):
            C(B.make_cfg(layers=layers, loop=loop))
    pc = C(B.make_cfg(layers=[B.retention(rot_dims=0)], loop=None))
    assert pc.layers[0].mixer.rot is None and pc.layer_runs() == [(0, None)]
    assert C(B.make_cfg(layers=[B.retention()], loop=(0, 1, 1))).layer_runs() == [(0, 0)]


def test_weight_mapping_fuses_pads_and_unrolls():
    A, C = pkg("_abi"), pkg("config")
    cfg = B.make_cfg()
    w = B.make_weights(cfg, 2)
    pc = B.product_config(cfg)
    items = {}
    for run, kind, t in pkg("weights").bofusun_weights(w, pc):
        assert (run, kind) not in items
        items[(run, kind)] = t
    assert torch.equal(items[(0, A.SW_EMBED_NORM)], 1.0 + w["embed.norm"]) and torch.equal(items[(2, A.SW_NORM_MIX_POST)], 1.0 + w["l2.norm1b"])
    # passes share tensors; the vectors of the passes go to the loop's first layer
    assert items[(1, A.SW_QKV)] is items[(3, A.SW_QKV)] and items[(2, A.SW_SIDE_A)] is items[(4, A.SW_SIDE_A)]
    assert torch.equal(items[(1, A.SW_LOOP_STEP)], w["loop.step"][0]) and torch.equal(items[(3, A.SW_LOOP_STEP)], w["loop.step"][1])
    assert not any((r, A.SW_LOOP_STEP) in items for r in (0, 2, 4, 5))
    p = "l0.mix.left."
    q, b, at = items[(0, A.SW_QKV)], items[(0, A.SW_QKV_BIAS)], 0
    for n in ("left.q", "left.k", "left.v", "right.in", "left.g"):
        t = w["l0.mix." + n]
        assert torch.equal(q[at:at + t.shape[0]], t), n
        assert torch.equal(b[at:at + t.shape[0]], w["l0.mix." + n + ".b"] if n[-1] in "qkv" else torch.zeros(t.shape[0])), n
        at += t.shape[0]
    assert at == q.shape[0] == b.shape[0]
    assert torch.equal(items[(0, A.SW_CONV)], torch.cat([w[p + n + ".conv"] for n in "qkv"]))
    table = items[(0, A.SW_DIST_BIAS)]
    assert table.shape == (4, 17)          # what the window shows
    for n in range(17):
        assert torch.equal(table[:, n], w[p + "rel"][O.bucket(n, 10, 40)])
    x, proj, dt = w["l0.mix.right.x"], items[(0, A.SW_SIDE_PROJ)], items[(0, A.SW_SIDE_DT)]
    assert proj.shape == (24, 28) and torch.equal(proj[:3], x[:3]) and torch.equal(proj[8:18], x[3:]) and float(proj[3:8].abs().max()) == 0.0
    assert dt.shape == (28, 8) and torch.equal(dt[:, :3], w["l0.mix.right.dt"]) and float(dt[:, 3:].abs().max()) == 0.0 and float(proj[18:].abs().max()) == 0.0
    assert torch.allclose(items[(0, A.SW_SIDE_A)].double(), -torch.exp(w["l0.mix.right.A_log"].double()))
    r = items[(5, A.SW_QKV)]
    assert torch.equal(r, torch.cat([w["l3.mix." + n] for n in "qkvg"])) and items[(5, A.SW_DECAY)].tolist() == cfg["layers"][3]["mixer"]["decay"]
    assert (5, A.SW_MLP_UP_BIAS) in items and (1, A.SW_NORM_MLP_PRE) not in items
    assert A.SW_QKV_BIAS not in A.SW_F32 and A.SW_DIST_BIAS in A.SW_F32 and A.SW_SIDE_A in A.SW_F32
    assert C.distance_entries(0, 40.0) == 41 and C.distance_entries(100, 40.0) == 41


def test_buckets_of_the_distance_table():
    C = pkg("config")
    for rows, far in ((10, 40), (16, 128), (32, 300), (2, 7), (6, 7)):
        got = [C.distance_bucket(n, rows, far) for n in range(2 * far)]
        assert got == [O.bucket(n, rows, far) for n in range(2 * far)]
        half = rows // 2
        assert got[:half] == list(range(half)) and got == sorted(got) and set(got[far:]) == {rows - 1} and got[half] == half
    assert [C.distance_bucket(n, 16, 128) for n in (8, 11, 12, 16, 32, 64, 127, 128)] == [8, 8, 9, 10, 12, 14, 15, 15]


def test_a_logit_row_does_not_depend_on_what_follows():
    cfg = B.make_cfg()
    w = B.make_weights(cfg, 3)
    ids = torch.randint(0, cfg["vocab"], (30,), generator=torch.Generator().manual_seed(1)).tolist()
    full = O.forward(cfg, w, ids)
    assert torch.allclose(O.forward(cfg, w, ids[:17]), full[:17], atol=1e-10)


def test_recurrences_carried_across_portions_equal_the_whole():
    g = torch.Generator().manual_seed(4)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    q, k, v, dec = r(23, 3, 5), r(23, 3, 5), r(23, 3, 4), torch.tensor([1.0, 0.9, 0.3], dtype=F64)
    whole, S_end = O.retention(q, k, v, dec)
    a, S = O.retention(q[:9], k[:9], v[:9], dec)
    b, S = O.retention(q[9:], k[9:], v[9:], dec, S)
    assert torch.allclose(torch.cat([a, b]), whole, atol=1e-12) and torch.allclose(S, S_end, atol=1e-12)
    t = 20      # the closed form of one row
    want = sum(dec[:, None] ** (t - j) * (q[t] * k[j]).sum(-1, keepdim=True) * v[j] for j in range(t + 1))
    assert torch.allclose(whole[t], want, atol=1e-10)
    x, dt, A, Bm, Cm, D = r(23, 6), r(23, 6).exp(), -r(6, 4).exp(), r(23, 4), r(23, 4), r(6)
    whole, _ = O.selective_scan(x, dt, A, Bm, Cm, D)
    a, S = O.selective_scan(x[:7], dt[:7], A, Bm[:7], Cm[:7], D)
    b, _ = O.selective_scan(x[7:], dt[7:], A, Bm[7:], Cm[7:], D, S)
    assert torch.allclose(torch.cat([a, b]), whole, atol=1e-12)
    u, cw = r(23, 6), r(6, 4)
    assert torch.allclose(torch.cat([O.causal_conv(u[:5], cw), O.causal_conv(u[5:], cw, history=u[2:5])]), O.causal_conv(u, cw), atol=1e-12)
    assert torch.allclose(O.causal_conv(u, cw)[0], u[0] * cw[:, 3])          # the last tap is the current token's


def test_window_edges_bias_and_cap_of_the_attention():
    T, w = 12, 5
    q, k = torch.zeros(T, 1, 2, dtype=F64), torch.zeros(T, 1, 2, dtype=F64)
    v = torch.eye(T, dtype=F64)[:, None, :]
    rel = torch.tensor([[0.5], [0.0], [-0.7], [0.2]], dtype=F64)
    p = O.biased_attention(q, k, v, 1.0, 3.0, rel, 6, w)[:, 0]
    assert torch.equal((p[11] > 0).nonzero().flatten(), torch.arange(7, 12)) and torch.equal((p[2] > 0).nonzero().flatten(), torch.arange(3))
    want = torch.softmax(torch.tensor([rel[O.bucket(11 - j, 4, 6), 0] for j in range(7, 12)], dtype=F64), 0)
    assert torch.allclose(p[11, 7:], want)
    q[:], k[8] = 10.0, 10.0         # a huge score saturates at the cap
    p = O.biased_attention(q, k, v, 1.0, 3.0, torch.zeros(4, 1, dtype=F64), 6, w)[:, 0]
    assert torch.allclose(p[11, 8] / p[11, 9], torch.tensor(math.exp(3.0), dtype=F64))


def test_what_a_pass_of_the_loop_takes():
    """With sublayers that return nothing (zero post-norm factor) the stream is what the loop adds: the embedding output once per
    pass after the first, and every pass's vector."""
    cfg = B.make_cfg(layers=[B.retention(), B.retention()], loop=(1, 2, 3))
    w = B.make_weights(cfg, 5)
    for n in ("l0.norm1b", "l1.norm1b"):
        w[n] = torch.full_like(w[n], -1.0)
    streams = []
    O.forward(cfg, w, [3, 7], streams)
    e = O.norm(w["embed"].double()[[3, 7]], w["embed.norm"].double(), 1e-5)
    st = w["loop.step"].double()
    assert len(streams) == 4 and O.passes(cfg) == [(0, None), (1, 0), (1, 1), (1, 2)]
    for got, want in zip(streams, (e, e + st[0], 2 * e + st[0] + st[1], 3 * e + st.sum(0))):
        assert torch.allclose(got, want, atol=1e-12)
