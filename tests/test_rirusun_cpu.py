"""Rirusun without a GPU: the registry and every part of the configuration, the unrolled layer list, the weight mapping (fusions,
zero biases, the expanded distance table, stacked gate matrices, the shared expert's gate row), and the oracle's own invariants
(causality, the recurrences' closed forms, the window's edges and kept first keys, the sink, the router's choices)."""
import math

import pytest
import torch

import rirusun_util as B
import stack_util as U
from conftest import pkg
from oracle import rirusun_oracle as O

F64 = torch.float64


def test_registry_reads_the_layer_list(tmp_path):
    cfg = B.make_cfg()
    path = str(tmp_path / "ckpt")
    U.write_checkpoint(path, cfg, B.make_weights(cfg, 1))
    C = pkg("config")
    pc = C.load_model_config(path)
    assert type(pc).__name__ == "RirusunConfig" and C.is_stack_config(pc) and pc.needs_state
    assert (pc.width, pc.vocab, pc.norm_eps, pc.embed_scale, pc.loop_start, pc.loop_stop, pc.loop_times) == (56, 110, 1e-5, 3.0, 1, 3, 2)
    assert pc.layer_runs() == [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (3, None)] and pc.n_layers == 6 and len(pc.layers) == 4
    la, pa, ml = (pc.layers[i].mixer for i in range(3))
    assert (la.heads, la.dim, la.rot_dim, la.vdim, la.kv_rank, la.scale, la.rot_half, la.sink, la.gate) == (3, 20, 12, 14, 28, 0.3, True, False, False)
    r = la.rot
    assert (r.base, r.dims, r.factor, r.original, r.fast, r.slow, r.scaled, r.kind) == (700.0, 12, 4.0, 48, 6.0, 0.5, True, "yarn")
    assert (pa.heads, pa.kv_heads, pa.dim, pa.vdim, pa.window, pa.keep_first, pa.scale, pa.bias_max) == (4, 2, 20, 12, 17, 3, 0.3, 40.0)
    assert pa.sink and pa.qk_norm and not pa.head_norm and pa.rot is None and not pa.bias
    s = pc.layers[1].side
    assert (s.inner, s.blocks, s.conv, s.kind) == (36, 3, 3, "lru") and pc.layers[1].side_mix == (0.7, 1.3)
    assert (ml.heads, ml.dim, ml.vdim, ml.gate_cap) == (3, 20, 12, 6.0)
    f = pc.layers[0].mlp
    assert (f.kind, f.ff, f.act, f.gated, f.experts, f.top, f.groups, f.keep, f.group_best) == ("moe", 24, "gelu_erf", False, 8, 3, 4, 2, 2)
    assert f.renorm and f.shared_gate and f.shared_ff == 20 and not f.weight_input
    f = pc.layers[1].mlp
    assert f.shared_ff == 0 and not f.shared_gate and (f.groups, f.keep) == (3, 2)
    f = pc.layers[2].mlp
    assert (f.groups, f.keep) == (1, 1) and pc.layers[3].mlp is None
    assert pc.kv_bytes_per_token() == 2 * (40 + 2 * 2 * 32 + 40) and pc.kv_bytes_per_token(True) == 2 * pc.kv_bytes_per_token()


def test_configuration_errors_and_defaults():
    C = pkg("config").RirusunConfig.from_dict
    for layers, loop in (([{"type": "retention", "mixer": {}, "mlp": None}], None), ([B.latent(rot_dim=7)], None), ([B.parallel(heads=3, kv_heads=2)], None),
                         ([B.parallel(width=35)], None), ([B.mlstm(mlp={"kind": "dense", "ff": 8})], None), ([B.mlstm(mlp=B.moe(groups=(3, 2)))], None),
                         ([B.mlstm(mlp=B.moe(top=5, groups=(4, 2)))], None), ([B.mlstm(mlp=B.moe(groups=(2, 3)))], None), ([B.mlstm(mlp=B.moe(top=9, groups=None))], None),
                         ([B.mlstm()], (0, 2, 2)), ([B.mlstm()], (0, 0, 2)), ([B.mlstm()], (0, 1, 0))):
        with pytest.raises(ValueError):
            C(B.make_cfg(layers=layers, loop=loop))
    pc = C(B.make_cfg(layers=[B.latent(rot_dim=0, scaling=None)], loop=None))
    assert pc.layers[0].mixer.rot is None and pc.layer_runs() == [(0, None)] and not pc.needs_state
    pc = C(B.make_cfg(layers=[B.latent(scaling=None)], loop=(0, 1, 1)))
    assert not pc.layers[0].mixer.rot.scaled and pc.layer_runs() == [(0, 0)]


def test_weight_mapping_fuses_stacks_and_unrolls():
    A, C = pkg("_abi"), pkg("config")
    cfg = B.make_cfg()
    w = B.make_weights(cfg, 2)
    pc = B.product_config(cfg)
    items = {}
    for run, kind, t in pkg("weights").rirusun_weights(w, pc):
        assert (run, kind) not in items
        items[(run, kind)] = t
    assert torch.equal(items[(0, A.SW_FINAL_NORM)], w["final.norm"]) and torch.equal(items[(0, A.SW_FINAL_NORM_BIAS)], w["final.norm.b"])
    assert items[(0, A.SW_FINAL_NORM_ALPHA)].shape == (1,) and torch.equal(items[(3, A.SW_NORM_MIX_PRE_BIAS)], w["l1.norm1.b"])
    assert items[(1, A.SW_QKV)] is items[(3, A.SW_QKV)] and items[(2, A.SW_EXPERT_DOWN)] is items[(4, A.SW_EXPERT_DOWN)]
    q, b, at = items[(1, A.SW_QKV)], items[(1, A.SW_QKV_BIAS)], 0
    for n in ("left.q", "left.k", "left.v", "right.x", "right.y"):
        t = w["l1.mix." + n]
        assert torch.equal(q[at:at + t.shape[0]], t), n
        assert torch.equal(b[at:at + t.shape[0]], w["l1.mix." + n + ".b"] if n[-1] in "xy" else torch.zeros(t.shape[0])), n
        at += t.shape[0]
    assert at == q.shape[0] == b.shape[0]
    table = items[(1, A.SW_DIST_BIAS)]
    assert table.shape == (4, 41)          # kept first keys lie at any distance
    for n in range(60):
        assert torch.equal(table[:, min(n, 40)], w["l1.mix.left.rel"][O.bucket(n, 10, 40)])
    gates, gb = items[(1, A.SW_SIDE_GATES)].view(3, 2, 12, 12), items[(1, A.SW_SIDE_GATES_BIAS)].view(3, 2, 12)
    for k, n in enumerate(("ra", "ri")):
        assert torch.equal(gates[:, k], w["l1.mix.right." + n]) and torch.equal(gb[:, k], w["l1.mix.right." + n + ".b"])
    assert torch.allclose(items[(1, A.SW_SIDE_DECAY)].double(), 8.0 * O.softplus(w["l1.mix.right.lam"].double()))
    assert torch.equal(items[(0, A.SW_ROUTER)], torch.cat([w["l0.mlp.router"], w["l0.mlp.shared.sg"]])) and items[(1, A.SW_ROUTER)].shape[0] == 6
    assert torch.equal(items[(0, A.SW_EXPERT_GATE_UP)][2 * 24:3 * 24], w["l0.mlp.e2.up"]) and (1, A.SW_SHARED_UP) not in items
    assert torch.equal(items[(0, A.SW_QKV)], torch.cat([w["l0.mix.q"], w["l0.mix.dkv"]]))
    uk = w["l0.mix.uk"].view(3, 20, 28)
    assert torch.equal(items[(0, A.SW_UK_T)].view(3, 28, 20), uk.transpose(1, 2))
    assert torch.equal(items[(2, A.SW_QKV)], torch.cat([w["l2.mix." + n] for n in "qkvg"]))
    assert A.SW_SIDE_GATES not in A.SW_F32 and A.SW_SIDE_DECAY in A.SW_F32 and A.SW_NORM_ALPHA in A.SW_F32
    assert C.distance_entries(17, 40.0, 3) == 41 and C.distance_entries(17, 40.0, 0) == 17


def test_a_logit_row_does_not_depend_on_what_follows():
    cfg = B.make_cfg()
    w = B.make_weights(cfg, 3)
    ids = torch.randint(0, cfg["vocab"], (30,), generator=torch.Generator().manual_seed(1)).tolist()
    full = O.forward(cfg, w, ids)
    assert torch.allclose(O.forward(cfg, w, ids[:17]), full[:17], atol=1e-10)


def test_closed_forms_of_the_recurrences():
    g = torch.Generator().manual_seed(4)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    u, ra, ri, lam = r(19, 6), torch.sigmoid(r(19, 6)), torch.sigmoid(r(19, 6)), r(6) - 3.0
    S = O.gated_lru(u, ra, ri, lam)
    la = -8.0 * ra * torch.log1p(torch.exp(lam))
    t = 15
    want = sum(torch.exp(la[j + 1:t + 1].sum(0)) * torch.sqrt(1 - torch.exp(2 * la[j])) * ri[j] * u[j] for j in range(t + 1))
    assert torch.allclose(S[t], want, atol=1e-12)
    assert torch.allclose(torch.cat([O.gated_lru(u[:7], ra[:7], ri[:7], lam), O.gated_lru(u[7:], ra[7:], ri[7:], lam, S[6])]), S, atol=1e-12)
    # matrix memory: the running maximum cancels up to the floor of the normaliser
    H, d, e, T = 2, 3, 4, 9
    q, k, v, li, lf = r(T, H, d), r(T, H, d), r(T, H, e), r(T, H), -O.softplus(-r(T, H))
    o = O.matrix_memory(q, k, v, li, lf)
    t = T - 1
    wgt = torch.stack([torch.exp(li[j] + lf[j + 1:t + 1].sum(0)) for j in range(t + 1)])                     # [T, H]
    dots = torch.stack([(k[j] * q[t]).sum(-1) for j in range(t + 1)])
    m = torch.zeros(H, dtype=F64)
    for j in range(T):
        m = torch.maximum(lf[j] + m, li[j])
    den = torch.maximum((wgt * dots).sum(0).abs(), torch.ones(H, dtype=F64)) + 1e-6 * torch.exp(m)
    assert torch.allclose(o[t], ((wgt * dots)[:, :, None] * v).sum(0) / den[:, None], atol=1e-10)


def test_window_edges_kept_keys_bias_and_sink():
    T, w, keep = 14, 5, 2
    q, k = torch.zeros(T, 1, 2, dtype=F64), torch.zeros(T, 1, 2, dtype=F64)
    v = torch.eye(T, dtype=F64)[:, None, :]
    rel = torch.tensor([[0.5], [0.0], [-0.7], [0.2]], dtype=F64)
    sink = torch.tensor([0.3], dtype=F64)
    p = O.kept_attention(q, k, v, 1.0, rel, 6, sink, w, keep)[:, 0]
    assert (p[13] > 0).nonzero().flatten().tolist() == [0, 1, 9, 10, 11, 12, 13] and (p[3] > 0).nonzero().flatten().tolist() == [0, 1, 2, 3]
    seen = [0, 1, 9, 10, 11, 12, 13]
    e = torch.exp(torch.tensor([float(rel[O.bucket(13 - j, 4, 6), 0]) for j in seen], dtype=F64))
    assert torch.allclose(p[13, seen], e / (e.sum() + math.exp(0.3)))
    assert torch.equal(O.visible(T, 0, 3), torch.ones(T, T).tril().bool())


def test_router_counts_groups_by_their_two_best_and_masks_negative_scores():
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    z = torch.zeros(1, 6, dtype=F64)
    # the best expert sits alone in its group; another group's two together beat it
    c = torch.tensor([0.3, -1.9, -0.1, -0.2, -1.5, -1.0], dtype=F64)
    ids, wts = O.route(z, c, r)
    assert ids.tolist() == [[2, 3]] and torch.allclose(wts, torch.full((1, 2), 0.5, dtype=F64))
    # every open choice score negative: the closed groups' larger ones still do not win
    c = torch.tensor([-0.9, -0.95, -0.55, -2.0, -3.0, -3.0], dtype=F64)
    assert O.route(z, c, r)[0].tolist() == [[0, 1]]
    ids, wts = O.route(torch.tensor([[2.0, 1.0, 0.0, -1.0]], dtype=F64), torch.zeros(4, dtype=F64), {"experts": 4, "top": 2})
    s = torch.sigmoid(torch.tensor([2.0, 1.0], dtype=F64))
    assert ids.tolist() == [[0, 1]] and torch.allclose(wts[0], s / s.sum())


def test_passes_of_the_loop_and_the_norm():
    cfg = B.make_cfg(layers=[B.mlstm(), B.mlstm()], loop=(1, 2, 3))
    assert O.passes(cfg) == [0, 1, 1, 1] and O.passes(B.make_cfg(layers=[B.mlstm()], loop=None)) == [0]
    w = B.make_weights(cfg, 5)
    for n in ("l0.mix.o", "l1.mix.o"):
        w[n] = torch.zeros_like(w[n])
    streams = []
    z = O.forward(cfg, w, [3, 7], streams)
    x = 3.0 * w["embed"].double()[[3, 7]]
    assert len(streams) == 4 and all(torch.equal(s, x) for s in streams)
    h = torch.tanh(w["final.norm.alpha"].double() * x) * w["final.norm"].double() + w["final.norm.b"].double()
    assert torch.allclose(z, h @ w["head"].double().T)
