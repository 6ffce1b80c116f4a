"""GPU parity of the Rirusun design against oracle/rirusun_oracle.py: every mechanism alone through its per-kernel entry point (with
inputs built so that a lost key, a window's edge, a sink, a stale state or a wrong tail shows), then whole models through the runner,
externally scheduled steps of the engine, and its own scheduler.  32-bit mode is held to the float64 oracle tightly; bf16 mode
within bf16 noise, and to itself across schedules."""
import numpy as np
import pytest
import torch

import rirusun_util as B
import stack_util as U
from conftest import pkg
from oracle import rirusun_oracle as O

pytestmark = pytest.mark.gpu
F32_TOL = 2e-5
DEV = "cuda"
_KEEP = []


def lib():
    return pkg("_abi").lib()


def check(rc):
    pkg("_abi").check(rc)


def dev(t, dtype=None):
    d = t.to(device=DEV, dtype=dtype or t.dtype).contiguous()
    _KEEP.append(d)
    del _KEEP[:-96]
    return d


def i32(x):
    return dev(torch.tensor(x, dtype=torch.int32))


def ptr(t):
    return None if t is None else t.data_ptr()


def sync():
    torch.cuda.synchronize()


def _prompt(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _adt(f32):
    return torch.float32 if f32 else torch.bfloat16


def _steps(lens, sizes, start_at):
    """Steps that carry several sequences side by side: per step the list of (name, first row, rows); sequence k starts at step
    start_at[k] and is cut by sizes[k]."""
    cuts = {}
    for k, n in lens.items():
        cuts[k], lo = [], 0
        for s in list(sizes[k]) + [n]:
            if lo < n:
                cuts[k].append((lo, min(s, n - lo)))
                lo += cuts[k][-1][1]
    n = max(start_at[k] + len(cuts[k]) for k in lens)
    steps = [[(k, *cuts[k][s - start_at[k]]) for k in lens if 0 <= s - start_at[k] < len(cuts[k])] for s in range(n)]
    return [s for s in steps if s]


def _meta(step):
    pos, rts, start = [], [], [0]
    for si, (_, lo, cnt) in enumerate(step):
        pos += list(range(lo, lo + cnt))
        rts += [si] * cnt
        start.append(start[-1] + cnt)
    return pos, rts, start


def _paged(T, bs, seed):
    nb = (T + bs - 1) // bs
    perm = torch.randperm(nb + 3, generator=torch.Generator().manual_seed(seed)).tolist()[:nb]
    return perm, [perm[t // bs] * bs + t % bs for t in range(T)], nb + 3


# ---- mechanisms alone ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("width", [40, 257, 1032])
@pytest.mark.parametrize("T", [5, 300])
def test_closing_sum_and_elementwise_norm(f32, width, T):
    """The opening norm alone; two weighted results, expert rows and a gated shared expert in one close; a close without a norm
    behind it; picked rows that leave the stream alone."""
    g = torch.Generator().manual_seed(width + T)
    adt, n = _adt(f32), 3
    tol = dict(atol=1e-5, rtol=1e-5) if f32 else dict(atol=1e-2, rtol=1e-2)
    r = lambda *s: torch.randn(*s, generator=g)
    x0, ya, yb, sh, parts = r(T, width), U.bf16_exact(2.0 * r(T, width)), U.bf16_exact(r(T, width)), U.bf16_exact(3.0 * r(T, width)), r(T, n, width)
    gate, alpha, w, b = torch.sigmoid(r(T)), torch.tensor([0.37]), 1 + 0.5 * r(width), r(width)
    D = lambda v: O.tanh_norm(v, alpha.double(), w.double(), b.double())
    x, out = dev(x0.clone()), torch.zeros(T, width, dtype=adt, device=DEV)
    yad, ybd, shd = dev(ya, adt), dev(yb, adt), dev(sh, adt)
    pd, gd, al, wd, bd = dev(parts), dev(gate), dev(alpha), dev(w), dev(b)

    def run(y=None, y2=None, p=0, s=None, gt=None, o=out, rows=None, R=T):
        check(lib().b200_tanh_close(f32, x.data_ptr(), ptr(y), 0.7, ptr(y2), -1.3, pd.data_ptr() if p else None, p, ptr(s), ptr(gt), al.data_ptr(),
                                    wd.data_ptr(), bd.data_ptr(), ptr(o), ptr(rows), R, width, None))
        sync()

    run()
    assert torch.equal(x.cpu(), x0) and torch.allclose(out.float().cpu().double(), D(x0.double()), **tol)
    run(yad, ybd, n, shd, gd)
    want = x0.double() + 0.7 * ya.double() - 1.3 * yb.double() + parts.double().sum(1) + gate.double()[:, None] * sh.double()
    assert torch.allclose(x.cpu().double(), want, atol=1e-5, rtol=1e-5) and torch.allclose(out.float().cpu().double(), D(want), **tol)
    x.copy_(x0.to(DEV))
    run(yad, None, n, shd, None, o=None)
    plain = x0.double() + 0.7 * ya.double() + parts.double().sum(1) + sh.double()
    assert torch.allclose(x.cpu().double(), plain, atol=1e-5, rtol=1e-5)
    x.copy_(x0.to(DEV))
    rows = [T - 1, 0, 3, 3]
    o3 = torch.zeros(4, width, dtype=adt, device=DEV)
    run(yad, ybd, n, shd, gd, o=o3, rows=i32(rows), R=4)
    assert torch.allclose(o3.float().cpu().double(), D(want[rows]), **tol) and torch.equal(x.cpu(), x0)


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,extra", [(4, 2, 20, 12, 8), (3, 1, 15, 7, 5), (16, 4, 128, 64, 0), (6, 6, 8, 36, 4)])
def test_whole_projection_norms_into_the_paged_cache(f32, heads, kv_heads, dim, vdim, extra):
    g = torch.Generator().manual_seed(dim)
    T, bs, eps, adt = 21, 8, 1e-3, _adt(f32)
    nq, nk, nv = heads * dim, kv_heads * dim, kv_heads * vdim
    fused = torch.randn(T, nq + nk + nv + extra, generator=g)
    fused[:, nq:nq + nk] *= 9.0                      # q and k have scales of their own
    fused = U.bf16_exact(fused)
    qw, kw = 1 + 0.3 * torch.randn(nq, generator=g), 1 + 0.3 * torch.randn(nk, generator=g)
    _, slots, nb = _paged(T, bs, 3)
    slots[5] = -1                                    # a row without a place in the cache
    kc, vc = torch.full((nb, kv_heads, bs, dim), 3.0, dtype=adt, device=DEV), torch.full((nb, kv_heads, bs, vdim), 3.0, dtype=adt, device=DEV)
    q = torch.zeros(T, nq, device=DEV)
    check(lib().b200_qk_norm_cache(f32, dev(fused, adt).data_ptr(), fused.shape[1], dev(qw).data_ptr(), dev(kw).data_ptr(), i32(slots).data_ptr(),
                                   q.data_ptr(), kc.data_ptr(), vc.data_ptr(), T, heads, kv_heads, dim, vdim, bs, eps, None))
    sync()
    x = fused.double()
    wq, wk, wv = O.unit_rms(x[:, :nq], eps) * qw.double(), O.unit_rms(x[:, nq:nq + nk], eps) * kw.double(), x[:, nq + nk:nq + nk + nv]
    assert torch.allclose(q.cpu().double(), wq, atol=1e-5, rtol=1e-5)
    rows = [t for t in range(T) if slots[t] >= 0]
    sl = torch.tensor([slots[t] for t in rows])
    tol = dict(atol=1e-5, rtol=1e-5) if f32 else dict(atol=1e-2, rtol=1e-2)
    assert torch.allclose(kc.float().cpu()[sl // bs, :, sl % bs].reshape(len(rows), nk).double(), wk[rows], **tol)
    assert torch.equal(vc.float().cpu()[sl // bs, :, sl % bs].reshape(len(rows), nv).double(), wv[rows])
    untouched = sorted(set(range(nb * bs)) - set(sl.tolist()))
    ut = torch.tensor(untouched)
    assert float((kc.float().cpu()[ut // bs, :, ut % bs] - 3.0).abs().max()) == 0.0


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("width", [28, 33, 520])
def test_convolution_without_activation_in_portions_with_dirty_slots(f32, taps, width):
    g = torch.Generator().manual_seed(taps * 10 + width)
    lens = {"a": 150, "b": 37, "c": 6}
    seqs = {k: U.bf16_exact(torch.randn(n, width, generator=g)) for k, n in lens.items()}
    cw, cb = U.bf16_exact(0.7 * torch.randn(width, taps, generator=g)), torch.randn(width, generator=g)
    want = {k: O.causal_conv(v.double(), cw.double(), cb.double()) for k, v in seqs.items()}
    slot_f = (taps - 1) * width + 4 + (-(taps - 1) * width) % 4
    state = dev(torch.full((4, slot_f), 9.0))
    slots, adt, off = {"a": 2, "b": 0, "c": 3}, _adt(f32), 4
    got = {k: torch.zeros(n, width) for k, n in lens.items()}
    cwd, cbd = dev(cw), dev(cb)
    sizes = {"a": [1, 2, 1, 1, 3, 100, 2, 1, 1, 1, 17], "b": [2, 1, 1, 16, 1, 1, 1, 1], "c": [1] * 6}
    for step in _steps(lens, sizes, {"a": 0, "b": 2, "c": 7}):
        pos, rts, start = _meta(step)
        rows = torch.cat([seqs[k][lo:lo + n] for k, lo, n in step])
        fused = torch.full((rows.shape[0], width + off + 4), 70.0)
        fused[:, off:off + width] = rows
        fd, T, S = dev(fused, adt), rows.shape[0], len(step)
        out = torch.zeros(T, width, dtype=adt, device=DEV)
        check(lib().b200_side_conv(f32, fd.data_ptr() + off * fd.element_size(), fused.shape[1], cwd.data_ptr(), cbd.data_ptr(), taps,
                                   state.data_ptr() if taps > 1 else None, slot_f, i32(pos).data_ptr(), i32(rts).data_ptr(), i32(start).data_ptr(),
                                   i32([slots[k] for k, _, _ in step]).data_ptr(), out.data_ptr(), T, S, width, int(T == S), None))
        sync()
        for si, (k, lo, n) in enumerate(step):
            got[k][lo:lo + n] = out[start[si]:start[si + 1]].float().cpu()
    for k in lens:
        assert torch.allclose(got[k].double(), want[k], **(dict(atol=1e-5, rtol=1e-5) if f32 else dict(atol=2e-2, rtol=1e-2))), k
    assert float((state[1] - 9.0).abs().max()) == 0.0


@pytest.mark.parametrize("y_f32,gated", [(1, 0), (0, 1), (0, 0)])
@pytest.mark.parametrize("T,heads,n_out,k", [(128, 2, 64, 16), (300, 3, 96, 48), (257, 2, 131, 80), (131, 1, 200, 272), (20, 3, 96, 48)])
def test_block_products_of_long_and_short_steps(y_f32, gated, T, heads, n_out, k):
    """Per-head (per-block) products on the tensor cores: tiles with ragged rows, outputs and inner chunks; the long form starts at 128 rows."""
    g = torch.Generator().manual_seed(T + k)
    x, w = U.bf16_exact(torch.randn(T, heads * k + 8, generator=g)), U.bf16_exact(torch.randn(heads, n_out, k, generator=g) * k ** -0.5)
    gate = U.bf16_exact(torch.randn(T, heads * n_out + 3, generator=g))
    ldy = heads * n_out + 5
    y = torch.full((T, ldy), 7.0, dtype=torch.float32 if y_f32 else torch.bfloat16, device=DEV)
    check(lib().b200_head_linear(0, y_f32, dev(x, torch.bfloat16).data_ptr(), heads * k + 8, k, dev(w, torch.bfloat16).data_ptr(), y.data_ptr(), ldy, n_out,
                                 dev(gate, torch.bfloat16).data_ptr() if gated else None, heads * n_out + 3, n_out, T, heads, n_out, k, None))
    sync()
    want = torch.einsum("thk,hok->tho", x[:, :heads * k].double().view(T, heads, k), w.double())
    if gated:
        want = want * torch.sigmoid(gate[:, :heads * n_out].double().view(T, heads, n_out))
    got = y.float().cpu().double()
    assert torch.allclose(got[:, :heads * n_out].view(T, heads, n_out), want, **(dict(atol=2e-5, rtol=1e-5) if y_f32 else dict(atol=1e-2, rtol=1e-2)))
    assert float((got[:, heads * n_out:] - 7.0).abs().max()) == 0.0


def _run_lru(f32, seqs, sizes, start_at, slots, bias, decay, blocks, slot_f, state):
    width = decay.shape[0]
    blk, adt = width // blocks, _adt(f32)
    bd, dd = dev(torch.stack([b.view(blocks, blk) for b in bias], 1).reshape(-1)), dev(decay)
    got = {k: torch.zeros(s["u"].shape) for k, s in seqs.items()}
    for step in _steps({k: s["u"].shape[0] for k, s in seqs.items()}, sizes, start_at):
        pos, _, start = _meta(step)
        cat = lambda n: torch.cat([seqs[k][n][lo:lo + c] for k, lo, c in step])
        T, S = len(pos), len(step)
        gates = torch.stack([cat("zr").view(T, blocks, blk), cat("zi").view(T, blocks, blk)], 2).reshape(T, 2 * width)
        ldy = width + (3 if width == 20 else 4)      # an odd row length keeps pairs of channels apart
        yy = torch.full((T, ldy), 50.0)
        yy[:, :width] = cat("y")
        out = torch.zeros(T, width, dtype=adt, device=DEV)
        check(lib().b200_gated_lru(f32, dev(cat("u"), adt).data_ptr(), dev(gates).data_ptr(), bd.data_ptr(), dd.data_ptr(), dev(yy, adt).data_ptr(), ldy,
                                   i32(pos).data_ptr(), i32(start).data_ptr(), i32([slots[k] for k, _, _ in step]).data_ptr(), state.data_ptr(), slot_f,
                                   out.data_ptr(), S, width, blocks, int(T == S), None))
        sync()
        for si, (k, lo, n) in enumerate(step):
            got[k][lo:lo + n] = out[start[si]:start[si + 1]].float().cpu()
    return got


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("width,blocks", [(36, 3), (17, 1), (130, 10), (256, 4), (5, 5), (34, 17), (20, 2)])
def test_gated_recurrent_unit_in_portions_with_three_sequences_and_dirty_slots(f32, width, blocks):
    """Decays from ones that wipe the state to ones that keep it for the whole sequence; portions from one row to several tiles of the
    scan, their ends on both sides of a tile's edge; the first input stands out, so that a state lost at an edge shows at the end."""
    g = torch.Generator().manual_seed(width)
    r = lambda *s: torch.randn(*s, generator=g)
    lens = {"a": 420, "b": 131, "c": 6}
    lam = torch.linspace(-14.0, 2.0, width)
    decay = (8.0 * O.softplus(lam.double())).float()
    bias = (r(width), r(width))
    seqs = {k: dict(u=U.bf16_exact(r(n, width)), y=U.bf16_exact(2.0 * r(n, width)), zr=2.0 * r(n, width), zi=2.0 * r(n, width)) for k, n in lens.items()}
    for s in seqs.values():
        s["u"][:2] *= 64.0
    want = {}
    for k, s in seqs.items():
        S = O.gated_lru(s["u"].double(), torch.sigmoid(s["zr"].double() + bias[0].double()), torch.sigmoid(s["zi"].double() + bias[1].double()), lam.double())
        want[k] = (S * O.gelu_tanh(s["y"].double()), S[-1])
    slot_f = width + 3
    slots = {"a": 4, "b": 1, "c": 0}
    cuts = {"portions": {"a": [1, 2, 128, 1, 127, 129, 3], "b": [127, 1, 1, 1], "c": [1] * 6}, "whole": {"a": [], "b": [], "c": []},
            "token by token": {"a": [386] + [1] * 34, "b": [100] + [1] * 31, "c": [1] * 6}}
    for name, sizes in cuts.items():
        state = dev(torch.full((5, slot_f), -3.0))
        got = _run_lru(f32, seqs, sizes, {"a": 0, "b": 1, "c": 2}, slots, bias, decay, blocks, slot_f, state)
        for k in lens:
            scale = float(want[k][1].abs().max())
            S_end = state[slots[k], :width].cpu().double()
            assert torch.allclose(S_end, want[k][1], atol=(2e-6 if f32 else 3e-6) * scale, rtol=2e-5), (name, k, float((S_end - want[k][1]).abs().max()))
            assert torch.allclose(got[k].double(), want[k][0], atol=1e-5 * scale if f32 else 4e-3 * scale, rtol=1e-4 if f32 else 1e-2), (name, k)
        assert float((state[2:4] + 3.0).abs().max()) == 0.0 and float((state[:, width:] + 3.0).abs().max()) == 0.0


def test_a_slow_decay_does_not_drift_over_thousands_of_rows():
    """Gates that never change and decays close to one: after 6000 rows the state still follows the closed form S_n = b (1 - a^n) /
    (1 - a) within fp32 rounding of one step (a decay rounded the same way at every row would be off a thousandfold)."""
    n, width = 6000, 32
    lam = torch.linspace(-13.0, -5.0, width, dtype=torch.float64)
    la = -8.0 * 0.5 * O.softplus(lam)
    b = torch.sqrt(-torch.expm1(2 * la)) * 0.5
    want = b * torch.expm1(n * la) / torch.expm1(la)
    for f32 in (1, 0):
        one = torch.ones(n, width)
        seqs = {"a": dict(u=one, y=one, zr=0 * one, zi=0 * one)}
        state = dev(torch.zeros(1, width))
        _run_lru(f32, seqs, {"a": [3000]}, {"a": 0}, {"a": 0}, (torch.zeros(width), torch.zeros(width)), (8.0 * O.softplus(lam)).float(), 4, width, state)
        assert torch.allclose(state[0].cpu().double(), want, rtol=1e-5), (f32, float((state[0].cpu().double() / want - 1).abs().max()))


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("heads,dim,rot_dim,kv_rank,scaled", [(3, 20, 12, 28, True), (2, 16, 32, 48, True), (1, 5, 6, 9, False)])
def test_latent_rows_and_rotated_queries_in_the_half_layout(f32, heads, dim, rot_dim, kv_rank, scaled):
    g = torch.Generator().manual_seed(dim)
    T, eps, adt = 60, 1e-4, _adt(f32)
    cfg = B.make_cfg(layers=[B.latent(heads=heads, dim=dim, rot_dim=rot_dim, kv_rank=kv_rank, scaling=B.YARN if scaled else None)], loop=None)
    m = cfg["layers"][0]["mixer"]
    spec = B.product_config(cfg).layers[0].mixer
    fused = U.bf16_exact(torch.randn(T, heads * (dim + rot_dim) + kv_rank + rot_dim, generator=g))
    nw = 1 + 0.3 * torch.randn(kv_rank, generator=g)
    slots = torch.randperm(T + 9, generator=g)[:T]
    krow = kv_rank + rot_dim
    q, cache = torch.full((T, heads, krow), 5.0, device=DEV), torch.full((T + 9, krow), 5.0, dtype=adt, device=DEV)
    check(lib().b200_latent_prep_half(f32, dev(fused, adt).data_ptr(), fused.shape[1], dev(nw).data_ptr(), i32(list(range(T))).data_ptr(),
                                      dev(slots.to(torch.int32)).data_ptr(), dev(spec.rot.table(64)).data_ptr(), rot_dim, 64, q.data_ptr(), cache.data_ptr(),
                                      T, heads, dim, rot_dim, kv_rank, eps, None))
    sync()
    x, pos = fused.double(), torch.arange(T)
    qr = O.rotate_half(x[:, :heads * (dim + rot_dim)].view(T, heads, dim + rot_dim)[..., dim:], pos, m["rot"])
    c = x[:, heads * (dim + rot_dim):]
    tol = dict(atol=2e-5, rtol=2e-5) if f32 else dict(atol=2e-2, rtol=1e-2)
    assert torch.allclose(q.cpu().double()[..., kv_rank:], qr, atol=2e-5, rtol=2e-5) and float((q[..., :kv_rank] - 5.0).abs().max()) == 0.0
    got = cache.float().cpu().double()[slots]
    assert torch.allclose(got[:, :kv_rank], O.unit_rms(c[:, :kv_rank], eps) * nw.double(), **tol)
    assert torch.allclose(got[:, kv_rank:], O.rotate_half(c[:, None, kv_rank:], pos, m["rot"])[:, 0], **tol)


@pytest.mark.parametrize("f32,linear", [(1, 0), (0, 0), (0, 1)])
@pytest.mark.parametrize("experts,top,groups,keep,width", [(8, 3, 4, 2, 64), (6, 2, 1, 1, 48), (64, 6, 8, 3, 128), (5, 5, 5, 5, 40), (12, 4, 3, 1, 33), (4, 1, 4, 2, 24)])
def test_router_by_pairs_of_scores_with_a_gate_row(f32, linear, experts, top, groups, keep, width):
    """Choice scores of either sign, groups decided by their two best (or their only one), weights that sum to one, the extra row."""
    linear = linear and width % 8 == 0           # the linear's widths
    g = torch.Generator().manual_seed(experts + width)
    T = 130
    x, wr = U.bf16_exact(torch.randn(T, width, generator=g)), U.bf16_exact(torch.randn(experts + 1, width, generator=g) * 2.0 * width ** -0.5)
    bias = 0.4 * torch.randn(experts, generator=g) - 0.5
    z = x.double() @ wr.double().T
    want_i, want_w = O.route(z[:, :experts], bias.double(), {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}})
    ids, wts, gate = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV), torch.zeros(T, device=DEV)
    logits = torch.zeros(T, experts + 1, device=DEV)
    for with_gate in (1, 0):
        check(lib().b200_moe_route_form(f32, dev(x, _adt(f32)).data_ptr(), dev(wr, torch.bfloat16).data_ptr(), dev(bias).data_ptr(), T, width, experts, top,
                                        groups, keep, 2, 1, gate.data_ptr() if with_gate else None, logits.data_ptr() if linear else None, ids.data_ptr(),
                                        wts.data_ptr(), None))
        sync()
        same = (ids.cpu().long().sort(1).values == want_i.sort(1).values).all(1)
        assert same.float().mean() > 0.98           # near-ties apart
        dense = torch.zeros(T, experts, dtype=torch.float64).scatter_(1, ids.cpu().long(), wts.cpu().double())
        want = torch.zeros(T, experts, dtype=torch.float64).scatter_(1, want_i, want_w)
        assert torch.allclose(dense[same], want[same], atol=1e-5)
    assert torch.allclose(gate.cpu().double(), torch.sigmoid(z[:, experts]), atol=1e-5)
    # the largest choice score sits in a group whose pair is weaker than another's: only one group may stay
    if groups > 1 and experts // groups > 1 and keep == 1:
        b2 = torch.full((experts,), -5.0)
        per = experts // groups
        b2[0], b2[per], b2[per + 1] = 5.0, 4.5, 4.5
        check(lib().b200_moe_route_form(f32, dev(x, _adt(f32)).data_ptr(), dev(wr, torch.bfloat16).data_ptr(), dev(b2).data_ptr(), T, width, experts, top, groups,
                                        keep, 2, 1, None, None, ids.data_ptr(), wts.data_ptr(), None))
        sync()
        assert (ids.cpu() // per == 1).all()


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("T,width,ff,experts,top", [(3, 40, 24, 5, 2), (70, 64, 40, 4, 3), (130, 128, 96, 8, 2), (5, 33, 7, 3, 3)])
def test_ungated_experts_with_exact_gelu(f32, T, width, ff, experts, top):
    g = torch.Generator().manual_seed(T + ff)
    A = pkg("_abi")
    x = U.bf16_exact(2.0 * torch.randn(T, width, generator=g))
    up, dn = U.bf16_exact(torch.randn(experts, ff, width, generator=g) * width ** -0.5), U.bf16_exact(torch.randn(experts, width, ff, generator=g) * ff ** -0.5)
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(T)])
    wts = torch.rand(T, top, generator=g)
    want = torch.stack([torch.stack([wts[t, j].double() * (dn[e].double() @ O.gelu_erf(up[e].double() @ x[t].double())) for j, e in enumerate(ids[t])])
                        for t in range(T)])
    parts = torch.zeros(T, top, width, device=DEV)
    ws = dev(torch.zeros(lib().b200_moe_workspace_bytes(T, top, experts, 0 if f32 else width, ff) // 4 + 4, dtype=torch.int32))
    check(lib().b200_moe_experts_form(f32, dev(x, _adt(f32)).data_ptr(), dev(up, torch.bfloat16).data_ptr(), dev(dn, torch.bfloat16).data_ptr(),
                                      dev(ids.to(torch.int32)).data_ptr(), dev(wts).data_ptr(), T, width, ff, experts, top, parts.data_ptr(), ws.data_ptr(), 0,
                                      A.ACT_GELU_ERF, 0, None))
    sync()
    assert torch.allclose(parts.cpu().double(), want, **(dict(atol=1e-5, rtol=1e-5) if f32 else dict(atol=2e-2, rtol=1e-2)))
    y = torch.zeros(T, ff, dtype=_adt(f32), device=DEV)      # the same activation in a dense linear's epilogue (the shared expert)
    lw = dev(torch.zeros(1 << 20, dtype=torch.int32))
    check(lib().b200_linear_bias_act(f32, 0, dev(x, _adt(f32)).data_ptr(), width, dev(up[0], torch.bfloat16).data_ptr(), None, y.data_ptr(), ff, T, ff, width,
                                     A.ACT_GELU_ERF, lw.data_ptr(), lw.numel() * 4, None))
    sync()
    assert torch.allclose(y.float().cpu().double(), O.gelu_erf(x.double() @ up[0].double().T), **(dict(atol=1e-5, rtol=1e-5) if f32 else dict(atol=2e-2, rtol=1e-2)))


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,keep,bs,T", [
    (4, 2, 24, 20, 33, 3, 16, 150), (3, 3, 32, 48, 64, 64, 64, 260), (5, 1, 48, 32, 70, 65, 32, 333), (2, 1, 16, 16, 1, 1, 16, 140), (6, 2, 64, 32, 128, 4, 128, 420),
    (5, 1, 40, 8, 0, 7, 8, 70), (4, 4, 16, 16, 20, 0, 16, 90), (2, 2, 16, 32, 8, 150, 16, 400)])
def test_windowed_attention_with_kept_keys_sink_and_far_bias(f32, heads, kv_heads, dim, vdim, window, keep, bs, T):
    """The oldest key of the window, the last kept key and the key after each limit carry a large entry that the last query asks for
    (those inside decide its output, those outside must not be seen); the distance bias is strong, differs by head and reaches the
    kept keys far away; the sinks take a large share.  All three kernels, the tensor-core one with and without splits."""
    g = torch.Generator().manual_seed(T + dim)
    scale, far, rows = 0.4, 0.6 * T, 12
    w = window or T
    q, k, v = (U.bf16_exact(torch.randn(T, h, d, generator=g)) for h, d in ((heads, dim), (kv_heads, dim), (kv_heads, vdim)))
    last = T - 1
    q[last, :, 0] = 6.0
    marks = set()
    if 0 < keep < last - w:
        k[keep - 1, :, 0], k[keep, :, 0] = 6.0, 40.0       # the last kept key, and the first that is not
        v[keep] = 30.0
        marks |= {"keep"}
    if w < T and last - w >= keep:
        k[last - w + 1, :, 0] = 6.0                        # the window's oldest key
        if last - w != keep:
            k[last - w, :, 0] = 40.0
        v[last - w] = 30.0
        marks |= {"window"}
    rel, sink = 2.0 * torch.randn(rows, heads, generator=g), 3.0 + torch.randn(heads, generator=g)
    d = lambda t: t.double()
    att = lambda w_, k_, s_: O.kept_attention(d(q), d(k), d(v), scale, d(rel), far, s_, w_, k_)
    want = att(window, keep, d(sink))
    # the construction bites: limits that are one token off, or a sink left out, change the last row by order one
    if "keep" in marks:
        assert float((att(window, keep + 1, d(sink))[last] - want[last]).abs().max()) > 0.1
        assert float((att(window, keep - 1, d(sink))[last] - want[last]).abs().max()) > 0.01
    if "window" in marks:
        assert float((att(window + 1, keep, d(sink))[last] - want[last]).abs().max()) > 0.1
    assert float((att(window, keep, torch.full((heads,), -1e30, dtype=torch.float64)) - want).abs().max()) > 0.1
    C = pkg("config")
    n_dist = C.distance_entries(window, far, keep)
    table = dev(rel[torch.tensor([C.distance_bucket(n, rows, far) for n in range(n_dist)])].T.contiguous())
    adt = _adt(f32)
    bt, slots, nb = _paged(T, bs, T)
    kc, vc = torch.full((nb, kv_heads, bs, dim), 3.0), torch.full((nb, kv_heads, bs, vdim), 3.0)
    for t in range(T):
        kc[slots[t] // bs, :, slots[t] % bs], vc[slots[t] // bs, :, slots[t] % bs] = k[t], v[t]
    kcd, vcd, qd, skd = dev(kc, adt), dev(vc, adt), dev(q.reshape(T, -1)), dev(sink)
    btd, ctx, rts, posd = i32(bt), i32(list(range(1, T + 1))), i32([0] * T), i32(list(range(T)))
    ws = dev(torch.zeros(lib().b200_paged_attn_anydim_workspace_bytes(T) // 4 + 4, dtype=torch.int32))
    forms = [(0, 1), (1, 1)]
    if not f32 and lib().b200_paged_attn_mma_supported(heads, kv_heads, dim, vdim):
        forms += [(2, 1), (2, 2), (2, 5)]
    for form, splits in forms:
        out = torch.zeros(T, heads * vdim, dtype=adt, device=DEV)
        part = dev(torch.zeros(T * heads * splits * (vdim + 2)))
        check(lib().b200_paged_attn_kept(f32, form, qd.data_ptr(), kcd.data_ptr(), vcd.data_ptr(), btd.data_ptr(), len(bt), rts.data_ptr(), ctx.data_ptr(),
                                         posd.data_ptr(), out.data_ptr(), T, heads, kv_heads, dim, vdim, bs, scale, window, keep, skd.data_ptr(),
                                         table.data_ptr(), n_dist, ws.data_ptr(), splits, part.data_ptr(), None))
        sync()
        tol = dict(atol=5e-5, rtol=5e-5) if f32 else dict(atol=6e-2, rtol=3e-2) if form == 2 else dict(atol=3e-2, rtol=2e-2)
        assert torch.allclose(out.float().cpu().double().view(T, heads, vdim), want, **tol), (form, splits)


# ---- whole models ----------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def model_a():
    cfg = B.make_cfg()
    return cfg, B.make_weights(cfg, 1)


ALONE = {
    "latent attention alone": ([B.latent()], None),
    "latent attention, plain frequencies, part of the shared key turning, with experts": ([B.latent(scaling=None, mlp=B.moe())], None),
    "latent attention without rotation": ([B.latent(rot_dim=0, scaling=None)], None),
    "the pair of mixers alone": ([B.parallel()], None),
    "the pair, one tap, as many key heads as heads, a window of one": ([B.parallel(kv_heads=4, conv=1, window=1, keep=1, mlp=B.moe())], None),
    "the pair, a window longer than the prompt, a table of two rows, one block": ([B.parallel(window=99, keep=0, rows=2, bias_max=7, blocks=1)], None),
    "the pair, more kept keys than the window": ([B.parallel(window=4, keep=11, mix=(1.0, 1.0))], None),
    "matrix memory alone": ([B.mlstm()], None),
    "matrix memory with experts, one group, no shared expert": ([B.mlstm(mlp=B.moe(groups=None, shared=None))], None),
    "every group kept": ([B.mlstm(mlp=B.moe(groups=(4, 4)))], None),
    "groups of one expert": ([B.mlstm(mlp=B.moe(experts=5, top=2, groups=(5, 3)))], None),
    "one pass": ([B.mlstm()], (0, 1, 1)),
    "the pair passed three times": ([B.parallel(mlp=B.moe())], (0, 1, 3)),
    "a loop in the middle": ([B.mlstm(), B.parallel(), B.latent(mlp=B.moe()), B.parallel(window=5)], (1, 3, 2)),
    "a loop to the end": ([B.latent(), B.mlstm()], (1, 2, 2)),
}


@pytest.mark.parametrize("which", list(ALONE))
def test_one_mechanism_models_and_their_streams_fp32(which):
    layers, loop = ALONE[which]
    cfg = B.make_cfg(width=64, layers=layers, loop=loop)
    w = B.make_weights(cfg, 4)
    ids = _prompt(cfg, 50, 1)
    r = B.make_runner(cfg, w, "float32")
    tap = r.set_stream_tap(True)
    got = U.replay(U.make_engine(r), [[("p", 50)]], {"p": ids})["p"]
    streams = []
    want = O.forward(cfg, w, ids, streams)
    assert U.rel_rms(got, want.numpy()).max() < F32_TOL
    L = len(streams)
    t = tap[:L * 50 * 64].view(L, 50, 64).cpu().double()
    assert torch.allclose(t, torch.stack(streams), atol=1e-4, rtol=1e-5)
    r.set_stream_tap(False)          # without the tap the last close runs over the logit rows alone
    assert U.rel_rms(U.replay(U.make_engine(r), [[("p", 50)]], {"p": ids})["p"], want.numpy()).max() < F32_TOL
    r.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("variant", ["odd sizes", "tensor-core sizes", "ones and equals"])
def test_other_sizes_and_constants(dtype, variant):
    """Widths and head sizes no vector access or TMA box fits; sizes that take every tensor-core path; constants that another
    model may make 1 or equal."""
    if variant == "odd sizes":
        cfg = B.make_cfg(width=101, vocab=131, eps=1e-3, loop=(0, 2, 3), scale=0.7, layers=[
            B.mlstm(heads=1, dim=34, vdim=50, cap=2.5, mlp=B.moe(experts=9, top=4, ff=13, groups=(3, 2), shared=11)),
            B.parallel(heads=6, kv_heads=3, dim=11, vdim=15, window=9, keep=2, bias_max=7, rows=6, width=39, blocks=13, conv=6, mix=(-0.4, 0.9)),
            B.latent(heads=5, dim=7, rot_dim=10, vdim=9, kv_rank=33, base=50.0, mlp=B.moe(experts=3, top=1, ff=20, groups=None))])
    elif variant == "tensor-core sizes":
        cfg = B.make_cfg(width=128, vocab=256, loop=(1, 2, 2), layers=[
            B.parallel(heads=4, kv_heads=2, dim=64, vdim=32, window=30, keep=4, width=256, blocks=4, conv=4, bias_max=24, rows=16,
                       mlp=B.moe(experts=8, top=2, ff=64, groups=(2, 1), shared=64)),
            B.latent(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, mlp=B.moe(experts=4, top=2, ff=128, groups=None, shared=128)),
            B.mlstm(heads=2, dim=64, vdim=64, mlp=B.moe(experts=16, top=4, ff=32, groups=(4, 2), shared=32)),
            B.parallel(heads=8, kv_heads=8, dim=16, vdim=16, window=64, keep=10, width=128, blocks=2, conv=3)])
    else:
        cfg = B.make_cfg(width=48, loop=(0, 1, 1), scale=1.0, layers=[
            B.latent(heads=1, dim=48, rot_dim=48, vdim=48, kv_rank=48, scale=1.0, mlp=B.moe(experts=1, top=1, ff=48, groups=(1, 1), shared=1)),
            B.parallel(heads=1, kv_heads=1, dim=48, vdim=48, window=2, keep=2, scale=1.0, bias_max=3, rows=2, width=48, blocks=48, conv=1, mix=(1.0, 1.0)),
            B.mlstm(heads=1, dim=48, vdim=48, cap=1.0)])
    w = B.make_weights(cfg, 6)
    ids = _prompt(cfg, 80, 2)
    want = O.forward(cfg, w, ids).numpy()
    r = B.make_runner(cfg, w, dtype)
    eng = U.make_engine(r)
    whole = U.replay(eng, [[("p", 80)]], {"p": ids})["p"]
    cut = U.replay(eng, [[("p", n)] for n in (2, 7, 1, 1, 16, 2, 20, 31)], {"p": ids})["p"]
    if dtype == "float32":
        assert U.rel_rms(whole, want).max() < F32_TOL and U.rel_rms(cut, want).max() < F32_TOL
    else:
        e = U.rel_rms(whole, want)
        assert np.median(e) < 0.03 and (e < 0.15).mean() > 0.9, (float(np.median(e)), float(e.max()))
        d = U.rel_rms(cut, whole)
        assert np.median(d) < 0.02 and (d < 0.15).mean() > 0.9, (float(np.median(d)), float(d.max()))
    r.close()


def test_every_schedule_gives_the_oracles_logits_fp32(model_a):
    """Prefill against token-by-token decoding, portions down to two tokens, unequal requests batched, a long decode tail that the
    windows pass over, blocks and state slots that are freed and taken again (12 blocks of 16 where the four requests need 22; four
    slots for the requests of all schedules)."""
    cfg, w = model_a
    prompts = {"a": _prompt(cfg, 70, 2), "b": _prompt(cfg, 37, 3), "c": _prompt(cfg, 3, 4), "d": _prompt(cfg, 110, 5)}
    want = {n: O.forward(cfg, w, p).numpy() for n, p in prompts.items()}
    r = B.make_runner(cfg, w, "float32", n_blocks=12, max_tokens=128)
    eng = U.make_engine(r)
    schedules = {
        "token by token": [[("c", 1)]] * 3 + [[("b", 1)]] * 37,
        "portions": [[("a", n)] for n in (2, 14, 1, 16, 17, 2, 2, 3, 13)],
        "prefill then a long decode": [[("d", 30)]] + [[("d", 1)]] * 80,
        "mixed": ([[("a", 33), ("c", 1)], [("c", 1), ("b", 2), ("a", 2)], [("b", 30), ("a", 1), ("c", 1)]] +
                  [[("a", 1), ("b", 1)]] * 5 + [[("a", 29)]] + [[("d", 64)], [("d", 2)], [("d", 44)]]),
    }
    for name, sched in schedules.items():
        got = U.replay(eng, sched, prompts)
        assert len(eng.blocks.free) == 12, name
        for n, l in got.items():
            assert l.shape[0] == len(prompts[n]), (name, n)
            assert U.rel_rms(l, want[n]).max() < F32_TOL, (name, n)
    r.close()


def test_a_request_left_out_of_steps_goes_on_where_it_stopped(model_a):
    cfg, w = model_a
    prompts = {"a": _prompt(cfg, 40, 21), "b": _prompt(cfg, 40, 22)}
    want = {n: O.forward(cfg, w, p).numpy() for n, p in prompts.items()}
    r = B.make_runner(cfg, w, "float32")
    sched = [[("a", 7)], [("b", 9)], [("b", 1)], [("a", 2), ("b", 1)], [("b", 29)], [("a", 31)]]
    got = U.replay(U.make_engine(r), sched, prompts)
    for n in prompts:
        assert U.rel_rms(got[n], want[n]).max() < F32_TOL, n
    r.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("through", ["latent key", "kept key", "recurrences"])
def test_the_first_tokens_decide_after_hundreds_of_steps(dtype, through):
    """A sequence of 600 tokens whose last logits still hang on the first tokens: through a latent key far away, through the kept
    first keys of a short window, or through recurrences that forget slowly.  Whole prompt, portions that cut pages and tiles, and
    decoding agree with the oracle."""
    layers = {"latent key": [B.latent(heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=32, scale=1.0, scaling=dict(factor=8.0, original=100, fast=4.0, slow=1.0))],
              "kept key": [B.parallel(heads=2, kv_heads=1, dim=16, vdim=16, window=20, keep=2, width=16, blocks=1, rows=8, bias_max=300, scale=0.5, mix=(1.0, 0.0))],
              "recurrences": [B.mlstm(heads=2, dim=32, vdim=32), B.parallel(heads=2, kv_heads=1, dim=16, vdim=16, window=20, keep=0, width=48, blocks=3)]}[through]
    cfg = B.make_cfg(width=64, vocab=90, loop=(0, len(layers), 2), layers=layers)
    w = B.make_weights(cfg, 12)
    if through == "kept key":
        w["l0.mix.left.rel"][-1] += 5.0        # the table's last row: what lies far away stands out
    if through == "recurrences":
        w["l0.mix.f.b"] = torch.full((2,), 6.0)
        w["l1.mix.right.lam"] = torch.full((48,), -11.0)
    w = {k: U.bf16_exact(v) for k, v in w.items()}
    ids = _prompt(cfg, 600, 9)
    want = O.forward(cfg, w, ids).numpy()
    other = O.forward(cfg, w, [(ids[0] + 1) % 90, (ids[1] + 7) % 90] + ids[2:]).numpy()
    assert U.rel_rms(other[-1:], want[-1:]).max() > 1e-3          # the start still shows at the end
    r = B.make_runner(cfg, w, dtype, max_tokens=640, max_model_len=640, block_size=64, n_blocks=10, max_logit_rows=640)
    eng = U.make_engine(r)
    whole = U.replay(eng, [[("p", 600)]], {"p": ids})["p"]
    cut = U.replay(eng, [[("p", n)] for n in (63, 2, 64, 129, 200, 110)] + [[("p", 1)]] * 32, {"p": ids})["p"]
    if dtype == "float32":
        assert U.rel_rms(whole, want).max() < F32_TOL and U.rel_rms(cut, want).max() < F32_TOL
    else:
        assert np.median(U.rel_rms(whole, want)) < 0.02 and U.rel_rms(whole, want).max() < 0.1
        assert np.median(U.rel_rms(cut, whole)) < 0.015 and U.rel_rms(cut, whole).max() < 0.1
    r.close()


def test_graph_replay_gives_the_same_logits_as_eager_steps(model_a):
    """Steps of equal shape replay one captured graph: sequence bounds, slots and positions must come from the step's device
    metadata, not from what was captured."""
    cfg, w = model_a
    prompts = {"a": _prompt(cfg, 40, 7), "b": _prompt(cfg, 40, 8)}
    sched = [[("a", 8), ("b", 8)]] * 3 + [[("a", 1), ("b", 1)]] * 16
    out = []
    for graphs in (False, True):
        r = B.make_runner(cfg, w, "float32", graphs=graphs)
        out.append(U.replay(U.make_engine(r), sched, prompts))
        r.close()
    for n in prompts:
        assert np.array_equal(out[0][n], out[1][n]), n


def test_passes_of_a_layer_share_one_upload(model_a):
    cfg, w = model_a
    r, once = B.make_runner(cfg, w, "float32"), B.make_runner(B.make_cfg(loop=None), w, "float32")
    assert r.cfg.n_layers == 6 and len(r.run_layers) == 6
    assert sum(t.numel() for t in r._weights) == sum(t.numel() for t in once._weights)
    assert r.state_bytes > once.state_bytes       # every pass has a state of its own
    r.close()
    once.close()


def test_bf16_mode_within_bf16_noise_and_equal_across_schedules(model_a):
    cfg, w = model_a
    prompts = {"a": _prompt(cfg, 70, 2), "b": _prompt(cfg, 37, 3)}
    want = {n: O.forward(cfg, w, p).numpy() for n, p in prompts.items()}
    r = B.make_runner(cfg, w, "bfloat16", n_blocks=12, max_tokens=128)
    eng = U.make_engine(r)
    whole = U.replay(eng, [[("a", 70)], [("b", 37)]], prompts)
    mixed = U.replay(eng, [[("a", 40), ("b", 2)], [("b", 20), ("a", 1)]] + [[("a", 1), ("b", 1)]] * 15 + [[("a", 14)]], prompts)
    for n in prompts:
        e = U.rel_rms(whole[n], want[n])
        assert np.median(e) < 0.03 and (e < 0.1).mean() > 0.9, (n, float(np.median(e)), float(e.max()))
        d = U.rel_rms(mixed[n], whole[n])
        assert np.median(d) < 0.02 and (d < 0.1).mean() > 0.9, (n, float(np.median(d)), float(d.max()))
    r.close()


def test_bf16_batches_of_long_portions_beside_single_tokens_equal_each_request_alone():
    """Sizes that take the tensor-core kernels: steps that carry portions of many rows, of a few rows and single decoded tokens of
    different sequences; every request gets what it gets alone, and the oracle's logits within bf16 noise."""
    cfg = B.make_cfg(width=128, vocab=150, loop=(0, 2, 2), layers=[
        B.latent(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, mlp=B.moe(experts=8, top=2, ff=64, groups=(2, 1), shared=64)),
        B.parallel(heads=4, kv_heads=2, dim=32, vdim=32, window=50, keep=4, width=128, blocks=4, conv=4),
        B.mlstm(heads=2, dim=64, vdim=48)])
    w = B.make_weights(cfg, 15)
    prompts = {"a": _prompt(cfg, 230, 1), "b": _prompt(cfg, 90, 2), "c": _prompt(cfg, 40, 3), "d": _prompt(cfg, 75, 4)}
    r = B.make_runner(cfg, w, "bfloat16", block_size=64, n_blocks=12, n_state_slots=5)
    eng = U.make_engine(r)
    mixed = U.replay(eng, [[("a", 70), ("c", 1)], [("b", 9), ("a", 1), ("c", 8)], [("c", 1), ("a", 130), ("b", 2), ("d", 64)],
                           [("a", 1), ("b", 64), ("d", 2), ("c", 1)]] + [[("a", 1), ("b", 1), ("c", 1), ("d", 1)]] * 9 + [[("a", 19), ("c", 20)], [("b", 6)]],
                     prompts)
    for n, p in prompts.items():
        alone = U.replay(eng, [[(n, len(p))]], prompts)[n]
        e, d = U.rel_rms(alone, O.forward(cfg, w, p).numpy()), U.rel_rms(mixed[n], alone)
        assert np.median(e) < 0.02 and (e < 0.08).mean() > 0.9, (n, float(np.median(e)), float(e.max()))
        assert np.median(d) < 0.02 and (d < 0.08).mean() > 0.9, (n, float(np.median(d)), float(d.max()))
    assert len(eng.blocks.free) == 12
    r.close()


def test_greedy_generation_through_the_engines_own_scheduler(model_a, tmp_path):
    """A checkpoint directory goes through the registry, the weight loader, LLMEngine.generate and the scheduler (which hands out
    blocks and state slots and overlaps steps); prompts of unequal length decode side by side."""
    cfg, w = model_a
    path = str(tmp_path / "ckpt")
    U.write_checkpoint(path, cfg, w)
    pc = pkg("config").load_model_config(path)
    assert type(pc).__name__ == "RirusunConfig"
    r = pkg("runner").make_runner(pc, dtype="float32", max_tokens=64, max_model_len=256, block_size=16, n_blocks=40, n_state_slots=4)
    r.load_weights(pkg("weights").load_safetensors_dir(path))
    eng = pkg("engine").LLMEngine(r, max_num_batched_tokens=64, max_num_seqs=8, max_model_len=256)
    assert eng.scheduler.max_seqs == 3          # bounded by the state slots
    prompts = [_prompt(cfg, 21, 11), _prompt(cfg, 5, 12), _prompt(cfg, 70, 13), _prompt(cfg, 9, 14)]
    got = eng.generate(prompts, max_tokens=14)
    for p, out in zip(prompts, got):
        ids = list(p)
        for tok in out:      # every emitted token is the oracle's arg-max, or within fp32 noise of it
            z = O.forward(cfg, w, ids)[-1]
            assert tok == int(z.argmax()) or float(z.max() - z[tok]) < 1e-3 * float(z.abs().max())
            ids.append(tok)
    r.close()


def test_samplers_and_log_probabilities_read_the_steps_logits(model_a):
    """Sampled requests go through the framework's samplers after the step: with top_k = 1 a request at temperature 0.9 emits the
    greedy tokens; the log-probabilities of the emitted tokens are the oracle's log-softmax (the samplers read bf16 logits); a
    plain greedy request in the same batch is untouched by its neighbours."""
    cfg, w = model_a
    E = pkg("engine")
    r = B.make_runner(cfg, w, "float32", max_tokens=64, max_model_len=256, n_blocks=40)
    eng = E.LLMEngine(r, max_num_batched_tokens=64, max_num_seqs=4, max_model_len=256)
    p = _prompt(cfg, 19, 55)      # its choices are no near-ties in bf16
    greedy = eng.generate([p], max_tokens=10)[0]
    reqs = [E.Request("s", list(p), max_tokens=10, ignore_eos=True, temperature=0.9, top_k=1, seed=5),
            E.Request("l", list(p), max_tokens=10, ignore_eos=True, logprobs=2),
            E.Request("g", list(p), max_tokens=10, ignore_eos=True)]
    for q in reqs:
        eng.add_request(q)
    while eng.has_work():
        eng.step()
    assert reqs[0].output_ids == greedy and reqs[1].output_ids == greedy and reqs[2].output_ids == greedy
    ids = list(p)
    for tok, (lp, top) in zip(reqs[1].output_ids, reqs[1].logprob_data):
        z = torch.log_softmax(O.forward(cfg, w, ids)[-1], -1)
        assert abs(lp - float(z[tok])) < 0.05 and top[0][0] == int(z.argmax())
        ids.append(tok)
    r.close()


def test_random_weights_of_the_benchmark_run(model_a):
    cfg, _ = model_a
    r = pkg("runner").make_runner(B.product_config(cfg), dtype="bfloat16", max_tokens=64, max_model_len=256, block_size=16, n_blocks=40, n_state_slots=4)
    r.init_random_weights(seed=3)
    eng = pkg("engine").LLMEngine(r, max_num_batched_tokens=64, max_num_seqs=3, max_model_len=256)
    out = eng.generate([_prompt(cfg, 30, 1), _prompt(cfg, 4, 2)], max_tokens=6)
    assert [len(o) for o in out] == [6, 6] and all(0 <= t < cfg["vocab"] for o in out for t in o)
    r.close()
