"""GPU parity of the Bofusun design against oracle/bofusun_oracle.py: every mechanism alone through its per-kernel entry point (with
inputs built so that a lost key, a window's edge, a stale state or a wrong tail shows), then whole models through the runner,
externally scheduled steps of the engine, and its own scheduler.  32-bit mode is held to the float64 oracle tightly; bf16 mode
within bf16 noise, and to itself across schedules."""
import numpy as np
import pytest
import torch

import bofusun_util as B
import stack_util as U
from conftest import pkg
from oracle import bofusun_oracle as O

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


def _portions(n, sizes):
    out, lo = [], 0
    for s in sizes:
        if lo >= n:
            break
        out.append((lo, min(s, n - lo)))
        lo += out[-1][1]
    if lo < n:
        out.append((lo, n - lo))
    return out


def _steps(lens, sizes, start_at):
    """Steps that carry several sequences side by side: per step the list of (name, first row, rows); sequence k starts at step
    start_at[k] and is cut by sizes[k]."""
    cuts = {k: _portions(lens[k], sizes[k]) for k in lens}
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


# ---- mechanisms alone ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("width", [40, 257, 1024])
@pytest.mark.parametrize("T", [7, 530])
def test_rms_row_pass_in_its_five_uses(f32, width, T):
    """Normed embedding kept aside and a pass's vector added; a plain close and open; two results averaged; a close that takes the
    embedding output and a vector ahead of the next norm, with the tap in between; picked rows that leave the stream alone."""
    g = torch.Generator().manual_seed(width + T)
    eps, adt = 1e-3, _adt(f32)
    tol = dict(atol=2e-5, rtol=2e-5) if f32 else dict(atol=3e-2, rtol=2e-2)
    r = lambda *s: torch.randn(*s, generator=g)
    raw, e, step = r(T, width), r(T, width), r(width)
    y, yb = U.bf16_exact(3.0 * r(T, width)), U.bf16_exact(0.2 * r(T, width))
    wa, wb, wp, wn = (1 + 0.3 * r(width) for _ in range(4))
    d = lambda t: t.double()
    N = lambda v, w: O.unit_rms(v, eps) * d(w)
    x, out, keep = dev(raw.clone()), torch.zeros(T, width, dtype=adt, device=DEV), torch.zeros(T, width, device=DEV)
    dv = {k: dev(v) for k, v in dict(e=e, step=step, wa=wa, wb=wb, wp=wp, wn=wn).items()}
    ya, ybd = dev(y, adt), dev(yb, adt)

    def run(yp, ybp, init=0, e_out=None, tap=None, e_=None, st=None, nxt=dv["wn"], rows=None, R=T, o=out):
        check(lib().b200_rms_sandwich(f32, x.data_ptr(), ptr(yp), ptr(ybp), dv["wa"].data_ptr() if ybp is not None else None,
                                      dv["wb"].data_ptr() if ybp is not None else None, dv["wp"].data_ptr(), init, ptr(e_out), ptr(tap), ptr(e_), ptr(st),
                                      ptr(nxt), ptr(o), ptr(rows), R, width, eps, None))
        sync()

    run(None, None, init=1, e_out=keep, st=dv["step"])
    e0 = N(d(raw), wp)
    assert torch.allclose(keep.cpu().double(), e0, atol=2e-5) and torch.allclose(x.cpu().double(), e0 + d(step), atol=2e-5)
    assert torch.allclose(out.float().cpu().double(), N(e0 + d(step), wn), **tol)
    xs = raw.clone()
    x.copy_(xs.to(DEV))
    run(ya, None)
    want = d(xs) + N(d(y), wp)
    assert torch.allclose(x.cpu().double(), want, atol=2e-5) and torch.allclose(out.float().cpu().double(), N(want, wn), **tol)
    x.copy_(xs.to(DEV))
    tap = torch.zeros(T, width, device=DEV)
    run(ya, ybd, tap=tap, e_=dv["e"], st=dv["step"])
    mix = 0.5 * (N(d(y), wa) + N(d(yb), wb))
    want = d(xs) + N(mix, wp)
    assert torch.allclose(tap.cpu().double(), want, atol=2e-5)
    assert torch.allclose(x.cpu().double(), want + d(e) + d(step), atol=2e-5)
    assert torch.allclose(out.float().cpu().double(), N(want + d(e) + d(step), wn), **tol)
    x.copy_(xs.to(DEV))
    rows = [T - 1, 0, 3]
    o3 = torch.zeros(3, width, dtype=adt, device=DEV)
    run(ya, ybd, rows=i32(rows), R=3, o=o3)
    assert torch.allclose(o3.float().cpu().double(), N(want[rows], wn), **tol) and torch.equal(x.cpu(), xs)


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("T,n_out,k", [(3, 40, 24), (130, 136, 64), (70, 50, 33), (300, 256, 128)])
def test_linear_with_bias_and_squared_relu(f32, T, n_out, k):
    g = torch.Generator().manual_seed(T + k)
    x, wt, b = (U.bf16_exact(torch.randn(*s, generator=g)) for s in ((T, k), (n_out, k), (n_out,)))
    adt = _adt(f32)
    ws = dev(torch.zeros(1 << 22, dtype=torch.int32))
    want = x.double() @ wt.double().T + b.double()
    for act, ref in ((-1, want), (pkg("_abi").ACT_RELU2, want.clamp(min=0) ** 2)):
        y = torch.zeros(T, n_out, dtype=adt, device=DEV)
        check(lib().b200_linear_bias_act(f32, 0, dev(x, adt).data_ptr(), k, dev(wt, torch.bfloat16).data_ptr(), dev(b, torch.bfloat16).data_ptr(), y.data_ptr(),
                                         n_out, T, n_out, k, act, ws.data_ptr(), ws.numel() * 4, None))
        sync()
        assert torch.allclose(y.float().cpu().double(), ref, atol=1e-3 if f32 else 0.05, rtol=1e-5 if f32 else 1e-2), act
    y = torch.zeros(T, n_out, device=DEV)      # unrounded rows
    check(lib().b200_linear_bias_act(f32, 1, dev(x, adt).data_ptr(), k, dev(wt, torch.bfloat16).data_ptr(), None, y.data_ptr(), n_out, T, n_out, k, -1,
                                     ws.data_ptr(), ws.numel() * 4, None))
    sync()
    assert torch.allclose(y.cpu().double(), want - b.double(), atol=1e-4, rtol=1e-5)


def _retention_want(fused, heads, dim, vdim, rot_dims, base, decay, eps):
    T = fused.shape[0]
    x = fused.double()
    hd, hv = heads * dim, heads * vdim
    pos = torch.arange(T)
    q = O.rotate_half(x[:, :hd].view(T, heads, dim), pos, rot_dims, base)
    k = O.rotate_half(x[:, hd:2 * hd].view(T, heads, dim), pos, rot_dims, base) * dim ** -0.5
    o, S = O.retention(q, k, x[:, 2 * hd:2 * hd + hv].reshape(T, heads, vdim), decay.double())
    return O.unit_rms(o, eps).reshape(T, hv) * O.silu(x[:, 2 * hd + hv:]), S


def _run_retention(form, f32, seqs, sizes, start_at, slots, heads, dim, vdim, rot_dims, base, decay, eps):
    """form 0: the step kernel alone; 1: step kernel for portions of up to 8 rows, chunks for longer ones; 2: chunks for all."""
    hv = heads * vdim
    off = 8
    slot_f = off + (heads * vdim * dim + 3) // 4 * 4 + 4
    state = dev(torch.full((max(slots.values()) + 2, slot_f), 7.0))
    rot = dev(pkg("config").RotarySpec(base=base, dims=rot_dims).table(1024)) if rot_dims else None
    adt = _adt(f32)
    dec = dev(decay)
    got = {k: torch.zeros(v.shape[0], hv) for k, v in seqs.items()}
    for step in _steps({k: v.shape[0] for k, v in seqs.items()}, sizes, start_at):
        pos, _, start = _meta(step)
        fused = dev(torch.cat([seqs[k][lo:lo + n] for k, lo, n in step]), adt)
        T, S, ld = fused.shape[0], len(step), fused.shape[1]
        out = torch.zeros(T, hv, dtype=adt, device=DEV)
        common = (fused.data_ptr(), ld, ptr(rot), rot_dims, 1, 1024, dec.data_ptr(), i32(pos).data_ptr(), i32(start).data_ptr(),
                  i32([slots[k] for k, _, _ in step]).data_ptr(), state.data_ptr() + 4 * off, slot_f, out.data_ptr())
        if form < 2:
            check(lib().b200_retention_step(f32, *common, S, heads, dim, vdim, eps, 8 if form else 0, None))
        if form:
            ws = dev(torch.full((lib().b200_retention_chunk_workspace_bytes(T, S, heads, dim, vdim) // 4,), float("nan")))
            check(lib().b200_retention_chunk(*common, T, S, heads, dim, vdim, eps, 8 if form == 1 else 0, ws.data_ptr(), None))
        sync()
        for si, (k, lo, n) in enumerate(step):
            got[k][lo:lo + n] = out[start[si]:start[si + 1]].float().cpu()
    S_end = {k: state[slots[k], off:off + heads * vdim * dim].cpu().double().view(heads, vdim, dim) for k in seqs}
    unused = [s for s in range(state.shape[0]) if s not in slots.values()]
    assert float((state[unused] - 7.0).abs().max()) == 0.0 and float((state[:, :off] - 7.0).abs().max()) == 0.0
    return got, S_end


RET_SHAPES = [(3, 20, 12, 16, 0), (1, 72, 40, 72, 0), (2, 33, 70, 2, 0), (2, 130, 8, 0, 0), (2, 80, 32, 48, 1), (3, 16, 48, 8, 1), (1, 128, 128, 64, 1),
              (2, 48, 80, 0, 1), (1, 32, 16, 32, 1)]


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("heads,dim,vdim,rot_dims,chunk", RET_SHAPES)
def test_retention_in_portions_with_three_sequences_and_dirty_slots(f32, heads, dim, vdim, rot_dims, chunk):
    """Decays from fast to none at all; portions of one row up to several chunks of 64, their ends on both sides of a chunk's edge; sequences that start
    later in slots full of other numbers.  The first tokens' values stand out, so that a state lost (or one decay too many) at a portion's
    or chunk's edge shows hundreds of rows later.  The final states are compared too."""
    g = torch.Generator().manual_seed(heads * 100 + dim)
    eps, base = 1e-5, 500.0
    decay = torch.tensor([1.0, 0.996, 0.8])[:heads] if heads > 1 else torch.tensor([0.998])
    lens = {"a": 203, "b": 65, "c": 9}
    width = 2 * heads * (dim + vdim)
    seqs = {k: torch.randn(n, width, generator=g) for k, n in lens.items()}
    for k in seqs:
        seqs[k][:2, 2 * heads * dim:2 * heads * dim + heads * vdim] *= 12.0
        seqs[k] = U.bf16_exact(seqs[k])
    want = {k: _retention_want(v, heads, dim, vdim, rot_dims, base, decay, eps) for k, v in seqs.items()}
    slots, start_at = {"a": 3, "b": 0, "c": 2}, {"a": 0, "b": 1, "c": 3}
    cuts = {"portions": {"a": [1, 2, 9, 64, 63, 1, 17, 40], "b": [2, 8, 1, 33, 21], "c": [1, 8]},
            "whole": {"a": [203], "b": [64], "c": [9]}, "token by token": {"a": [170] + [1] * 33, "b": [40] + [1] * 25, "c": [1] * 9}}
    forms = [0] + ([1, 2] if chunk and not f32 else [])
    for form in forms:
        for name, sizes in cuts.items():
            got, S = _run_retention(form, f32, seqs, sizes, start_at, slots, heads, dim, vdim, rot_dims, base, decay, eps)
            for k in seqs:
                assert torch.allclose(S[k].transpose(1, 2), want[k][1], atol=2e-4 if form else 3e-5, rtol=3e-4 if form else 1e-4), (form, name, k)
                tol = dict(atol=3e-5, rtol=1e-4) if f32 else dict(atol=2e-2, rtol=1e-2)      # bf16: the output's own rounding
                assert torch.allclose(got[k].double(), want[k][0], **tol), (form, name, k, float((got[k].double() - want[k][0]).abs().max()))
    if chunk:
        assert lib().b200_retention_chunk_supported(dim, vdim)


def test_retention_with_pairs_of_neighbours_turning():
    """The other pair layout of the step kernel (dimension 2i with 2i + 1)."""
    g = torch.Generator().manual_seed(5)
    heads, dim, vdim, n = 2, 12, 8, 11
    fused = U.bf16_exact(torch.randn(n, 2 * heads * (dim + vdim), generator=g))
    perm = torch.tensor([0, 2, 4, 6, 1, 3, 5, 7, 8, 9, 10, 11])       # half layout <- pair layout over 8 turning dimensions
    half = fused.clone()
    for h in range(2 * heads):
        half[:, h * dim:(h + 1) * dim] = fused[:, h * dim:(h + 1) * dim][:, perm]
    want, _ = _retention_want(half, heads, dim, vdim, 8, 100.0, torch.tensor([0.9, 0.99]), 1e-5)
    rot = dev(pkg("config").RotarySpec(base=100.0, dims=8).table(64))
    out, state = torch.zeros(n, heads * vdim, device=DEV), torch.zeros(heads * dim * vdim, device=DEV)
    check(lib().b200_retention_step(1, dev(fused).data_ptr(), fused.shape[1], rot.data_ptr(), 8, 0, 64, dev(torch.tensor([0.9, 0.99])).data_ptr(),
                                    i32(list(range(n))).data_ptr(), i32([0, n]).data_ptr(), i32([0]).data_ptr(), state.data_ptr(), state.numel(),
                                    out.data_ptr(), 1, heads, dim, vdim, 1e-5, 0, None))
    sync()
    assert torch.allclose(out.cpu().double(), want, atol=3e-5)


def _paged(T, bs, seed):
    nb = (T + bs - 1) // bs
    perm = torch.randperm(nb + 3, generator=torch.Generator().manual_seed(seed)).tolist()[:nb]
    return perm, [perm[t // bs] * bs + t % bs for t in range(T)], nb + 3


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("taps_a,taps_x", [(1, 4), (2, 1), (3, 2), (4, 3), (0, 5), (7, 9)])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,inner", [(4, 2, 20, 12, 28), (3, 1, 10, 14, 33)])
def test_convolved_inputs_in_portions_with_three_sequences_and_dirty_slots(f32, taps_a, taps_x, heads, kv_heads, dim, vdim, inner):
    """q, k, v without and x with bias and activation; portions shorter and longer than the tails, runs that start in the middle of a
    sequence, steps of one row each (which shift the tails in place), cache rows at shuffled slots."""
    g = torch.Generator().manual_seed(taps_a * 10 + taps_x)
    n_a, bs = heads * dim + kv_heads * (dim + vdim), 8
    lens = {"a": 190, "b": 37, "c": 6}
    seqs = {k: U.bf16_exact(torch.randn(n, n_a + inner, generator=g)) for k, n in lens.items()}
    wa, wx, bx = U.bf16_exact(0.6 * torch.randn(n_a, max(taps_a, 1), generator=g)), U.bf16_exact(0.6 * torch.randn(inner, taps_x, generator=g)), \
        torch.randn(inner, generator=g)
    want = {k: (v[:, :n_a].double() if taps_a == 0 else O.causal_conv(v[:, :n_a].double(), wa.double()),
                O.silu(O.causal_conv(v[:, n_a:].double(), wx.double(), bx.double()))) for k, v in seqs.items()}
    ta, tx = max(taps_a - 1, 0) * n_a, (taps_x - 1) * inner
    up4 = lambda v: (v + 3) // 4 * 4
    slot_f = up4(ta) + up4(tx) + 4
    state = dev(torch.full((4, slot_f), 9.0))
    pa, px = state.data_ptr() if taps_a > 1 else None, state.data_ptr() + 4 * up4(ta) if taps_x > 1 else None
    slots = {"a": 2, "b": 0, "c": 3}
    adt, es = _adt(f32), 4 if f32 else 2
    tables = {k: _paged(n, bs, n) for k, n in lens.items()}
    base, nb = {}, 0
    for k in lens:
        base[k] = nb
        nb += tables[k][2]
    kc = torch.full((nb, kv_heads, bs, dim), 3.0, dtype=adt, device=DEV)
    vc = torch.full((nb, kv_heads, bs, vdim), 3.0, dtype=adt, device=DEV)
    got = {k: (torch.zeros(n, n_a), torch.zeros(n, inner)) for k, n in lens.items()}
    wad, wxd, bxd = dev(wa), dev(wx), dev(bx)
    sizes = {"a": [1, 2, 1, 1, 3, 130, 2, 1, 1, 1, 17], "b": [2, 1, 1, 16, 1, 1, 1, 1], "c": [1, 1, 1, 1, 1, 1]}
    nq, nk = heads * dim, kv_heads * dim
    for step in _steps(lens, sizes, {"a": 0, "b": 2, "c": 7}):
        pos, rts, start = _meta(step)
        fused = dev(torch.cat([seqs[k][lo:lo + n] for k, lo, n in step]), adt)
        T, S, ld = fused.shape[0], len(step), fused.shape[1]
        one = int(T == S)
        sl = i32([base[k] * bs + tables[k][1][t] for k, lo, n in step for t in range(lo, lo + n)])
        posd, rtsd, std, sld = i32(pos), i32(rts), i32(start), i32([slots[k] for k, _, _ in step])
        q, xc = torch.zeros(T, nq, device=DEV), torch.zeros(T, inner, dtype=adt, device=DEV)
        check(lib().b200_conv_inputs(f32, fused.data_ptr(), ld, wad.data_ptr() if taps_a else None, taps_a, pa, wxd.data_ptr(), bxd.data_ptr(), taps_x, px,
                                     slot_f, posd.data_ptr(), rtsd.data_ptr(), std.data_ptr(), sld.data_ptr(), sl.data_ptr(), q.data_ptr(), kc.data_ptr(),
                                     vc.data_ptr(), xc.data_ptr(), T, heads, kv_heads, dim, vdim, inner, bs, one, None))
        if not one and taps_a > 1:
            check(lib().b200_delta_tails(f32, fused.data_ptr(), ld, posd.data_ptr(), std.data_ptr(), sld.data_ptr(), pa, slot_f, S, n_a, taps_a, None))
        if not one and taps_x > 1:
            check(lib().b200_delta_tails(f32, fused.data_ptr() + n_a * es, ld, posd.data_ptr(), std.data_ptr(), sld.data_ptr(), px, slot_f, S, inner, taps_x,
                                         None))
        sync()
        for si, (k, lo, n) in enumerate(step):
            got[k][0][lo:lo + n, :nq] = q[start[si]:start[si + 1]].cpu()
            got[k][1][lo:lo + n] = xc[start[si]:start[si + 1]].float().cpu()
    tol = dict(atol=1e-5, rtol=1e-5) if f32 else dict(atol=2e-2, rtol=1e-2)
    for k, n in lens.items():
        assert torch.allclose(got[k][0][:, :nq].double(), want[k][0][:, :nq], atol=1e-5), k
        assert torch.allclose(got[k][1].double(), want[k][1], **tol), k
        sl = torch.tensor([base[k] * bs + s for s in tables[k][1]])
        kk = kc.float().cpu()[sl // bs, :, sl % bs].reshape(n, nk).double()
        vv = vc.float().cpu()[sl // bs, :, sl % bs].reshape(n, kv_heads * vdim).double()
        assert torch.allclose(kk, want[k][0][:, nq:nq + nk], **tol) and torch.allclose(vv, want[k][0][:, nq + nk:], **tol), k
    assert float((state[1] - 9.0).abs().max()) == 0.0


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("inner,state,rank", [(28, 5, 3), (130, 16, 8), (33, 1, 1), (20, 24, 5), (12, 70, 2), (9, 130, 4), (260, 4, 16), (40, 8, 2)])
def test_selective_scan_in_portions_with_three_sequences_and_dirty_slots(f32, inner, state, rank):
    """Lane groups of every size; step sizes from almost none to ones that wipe the state; a first token whose input stands out."""
    g = torch.Generator().manual_seed(inner + state)
    lens = {"a": 75, "b": 33, "c": 5}
    A = -torch.exp(torch.randn(inner, state, generator=g) - 1.0)
    D, dtb = torch.randn(inner, generator=g), torch.randn(inner, generator=g) - 1.0
    seqs = {k: dict(x=U.bf16_exact(torch.randn(n, inner, generator=g)), f=U.bf16_exact(torch.randn(n, 2 * state, generator=g)),
                    dt=2.0 * torch.randn(n, inner, generator=g), z=U.bf16_exact(torch.randn(n, inner, generator=g))) for k, n in lens.items()}
    for s in seqs.values():
        s["x"][0] *= 16.0
    want = {}
    for k, s in seqs.items():
        y, S = O.selective_scan(s["x"].double(), O.softplus(s["dt"].double() + dtb.double()), A.double(), s["f"][:, :state].double(),
                                s["f"][:, state:].double(), D.double())
        want[k] = (y * O.silu(s["z"].double()), S)
    adt = _adt(f32)
    slot_f = inner * state + 5
    st = dev(torch.full((5, slot_f), -3.0))
    slots, got = {"a": 4, "b": 1, "c": 0}, {k: torch.zeros(n, inner) for k, n in lens.items()}
    ldbc, off = 2 * state + 11, 7
    sizes = {"a": [1, 2, 16, 1, 17, 33], "b": [32, 1], "c": [1] * 5}      # the last step of c and its like bring one row each
    Ad, Dd, dtbd = dev(A), dev(D), dev(dtb)
    for step in _steps(lens, sizes, {"a": 0, "b": 1, "c": 2}):
        pos, _, start = _meta(step)
        cat = lambda n: torch.cat([seqs[k][n][lo:lo + c] for k, lo, c in step])
        T, S = len(pos), len(step)
        bc = torch.full((T, ldbc), 50.0)
        bc[:, off:off + 2 * state] = cat("f")
        zz = torch.full((T, inner + 3), 50.0)
        zz[:, :inner] = cat("z")
        out = torch.zeros(T, inner, dtype=adt, device=DEV)
        check(lib().b200_selective_scan(f32, dev(cat("x"), adt).data_ptr(), dev(bc, adt).data_ptr(), ldbc, off, dev(cat("dt")).data_ptr(), dtbd.data_ptr(),
                                        Ad.data_ptr(), Dd.data_ptr(), dev(zz, adt).data_ptr(), inner + 3, i32(pos).data_ptr(), i32(start).data_ptr(),
                                        i32([slots[k] for k, _, _ in step]).data_ptr(), st.data_ptr(), slot_f, out.data_ptr(), S, inner, state, int(T == S), None))
        sync()
        for si, (k, lo, n) in enumerate(step):
            got[k][lo:lo + n] = out[start[si]:start[si + 1]].float().cpu()
    for k in lens:
        scale = float(want[k][0].abs().max())
        assert torch.allclose(got[k].double(), want[k][0], atol=2e-6 * scale + 2e-5 if f32 else 4e-3 * scale, rtol=1e-4 if f32 else 1e-2), k
        S_end = st[slots[k], :inner * state].cpu().double().view(inner, state)
        assert torch.allclose(S_end, want[k][1], atol=1e-4, rtol=1e-4), k
    assert float((st[2:4] + 3.0).abs().max()) == 0.0 and float((st[:, inner * state:] + 3.0).abs().max()) == 0.0


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,bs,T", [(4, 2, 24, 20, 33, 16, 150), (3, 3, 32, 48, 64, 64, 200), (5, 1, 48, 32, 70, 32, 200),
                                                                 (2, 1, 16, 16, 1, 16, 40), (6, 2, 64, 32, 128, 128, 300), (5, 1, 40, 8, 0, 8, 70)])
def test_capped_distance_biased_windowed_attention_with_decisive_keys(f32, heads, kv_heads, dim, vdim, window, bs, T):
    """Keys just inside and just outside the window carry a large entry that the last query asks for (the one inside decides that
    query's output, the one outside must not be seen); the distance bias is strong and differs by head; the cap bends the large
    scores; one gate per head.  All three kernels, the tensor-core one with and without splits."""
    g = torch.Generator().manual_seed(T + dim)
    scale, cap, far, rows = 0.4, 6.0, 0.7 * (window or T), 12
    w = window or T
    q, k, v = (U.bf16_exact(torch.randn(T, h, d, generator=g)) for h, d in ((heads, dim), (kv_heads, dim), (kv_heads, vdim)))
    last = T - 1
    q[last, :, 0] = 6.0
    if w < T:
        k[last - w + 1, :, 0] = 6.0        # the oldest key the last query sees
        k[last - w, :, 0] = 40.0           # one token further: outside
        v[last - w] = 30.0
    rel = 2.0 * torch.randn(rows, heads, generator=g)
    gate = U.bf16_exact(torch.randn(T, heads + 3, generator=g))
    d = lambda t: t.double()
    sig = torch.sigmoid(d(gate[:, :heads]))[:, :, None]
    want = O.biased_attention(d(q), d(k), d(v), scale, cap, d(rel), far, w) * sig
    if 1 < w < T:      # the construction bites: a window one token wider or narrower changes the last row by order one
        for other in (w - 1, w + 1):
            assert float((O.biased_attention(d(q), d(k), d(v), scale, cap, d(rel), far, other)[last] * sig[last] - want[last]).abs().max()) > 0.1
    C = pkg("config")
    n_dist = C.distance_entries(window, far)
    table = dev(rel[torch.tensor([C.distance_bucket(n, rows, far) for n in range(n_dist)])].T.contiguous())
    adt = _adt(f32)
    bt, slots, nb = _paged(T, bs, T)
    kc, vc = torch.full((nb, kv_heads, bs, dim), 3.0), torch.full((nb, kv_heads, bs, vdim), 3.0)
    for t in range(T):
        kc[slots[t] // bs, :, slots[t] % bs], vc[slots[t] // bs, :, slots[t] % bs] = k[t], v[t]
    kcd, vcd, qd, gd = dev(kc, adt), dev(vc, adt), dev(q.reshape(T, -1)), dev(gate, adt)
    btd, ctx, rts, posd = i32(bt), i32(list(range(1, T + 1))), i32([0] * T), i32(list(range(T)))
    ws = dev(torch.zeros(lib().b200_paged_attn_anydim_workspace_bytes(T) // 4 + 4, dtype=torch.int32))
    forms = [(0, 1), (1, 1)]
    if not f32 and lib().b200_paged_attn_mma_supported(heads, kv_heads, dim, vdim):
        forms += [(2, 1), (2, 3)]
    for form, splits in forms:
        out = torch.zeros(T, heads * vdim, dtype=adt, device=DEV)
        part = dev(torch.zeros(T * heads * splits * (vdim + 2)))
        check(lib().b200_paged_attn_biased(f32, form, qd.data_ptr(), kcd.data_ptr(), vcd.data_ptr(), btd.data_ptr(), len(bt), rts.data_ptr(), ctx.data_ptr(),
                                           posd.data_ptr(), out.data_ptr(), T, heads, kv_heads, dim, vdim, bs, scale, window, cap, table.data_ptr(), n_dist,
                                           gd.data_ptr(), heads + 3, ws.data_ptr(), splits, part.data_ptr(), None))
        sync()
        tol = dict(atol=5e-5, rtol=5e-5) if f32 else dict(atol=6e-2, rtol=3e-2) if form == 2 else dict(atol=3e-2, rtol=2e-2)
        assert torch.allclose(out.float().cpu().double().view(T, heads, vdim), want, **tol), (form, splits)


# ---- whole models ----------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def model_a():
    cfg = B.make_cfg()
    return cfg, B.make_weights(cfg, 1)


ALONE = {
    "retention alone": ([B.retention()], None),
    "retention, part of each head turning, with a feed-forward": ([B.retention(rot_dims=8, mlp=B.dense(17))], None),
    "retention without rotation": ([B.retention(rot_dims=0)], None),
    "the pair of mixers alone": ([B.parallel()], None),
    "the pair, one tap, as many key heads as heads, a window of one": ([B.parallel(kv_heads=4, conv=1, conv2=1, window=1, mlp=B.dense())], None),
    "the pair, a window longer than the prompt, a table of two rows": ([B.parallel(window=99, rows=2, bias_max=7)], None),
    "one pass with its vector": ([B.retention()], (0, 1, 1)),
    "the pair passed three times": ([B.parallel(mlp=B.dense())], (0, 1, 3)),
    "a loop in the middle": ([B.retention(), B.parallel(), B.retention(mlp=B.dense()), B.parallel(window=5)], (1, 3, 2)),
    "a loop to the end": ([B.retention(), B.parallel()], (1, 2, 2)),
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
    r.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("variant", ["odd sizes", "tensor-core sizes", "ones and equals"])
def test_other_sizes_and_constants(dtype, variant):
    """Widths and head sizes no vector access or TMA box fits; sizes that take every tensor-core path; constants that another
    model may make 1 or equal."""
    if variant == "odd sizes":
        cfg = B.make_cfg(width=101, vocab=131, eps=1e-3, loop=(0, 2, 3), layers=[
            B.retention(heads=1, dim=34, vdim=50, rot_dims=10, mlp=B.dense(43)),
            B.parallel(heads=6, kv_heads=3, dim=10, vdim=15, window=9, conv=5, softcap=1.5, bias_max=7, rows=6, inner=37, state=18, dt_rank=11, conv2=6),
            B.parallel(heads=5, kv_heads=1, dim=7, vdim=9, window=31, conv=2, bias_max=100, rows=32, inner=21, state=33, dt_rank=1, conv2=4, mlp=B.dense(20))])
    elif variant == "tensor-core sizes":
        cfg = B.make_cfg(width=128, vocab=256, loop=(1, 2, 2), layers=[
            B.parallel(heads=4, kv_heads=2, dim=64, vdim=32, window=30, conv=4, inner=256, state=16, dt_rank=8, conv2=4, bias_max=24, rows=16, mlp=B.dense(256)),
            B.retention(heads=2, dim=64, vdim=64, rot_dims=64),
            B.retention(heads=4, dim=32, vdim=48, rot_dims=16, mlp=B.dense(64)),
            B.parallel(heads=8, kv_heads=8, dim=16, vdim=16, window=64, inner=128, state=32, dt_rank=16, conv2=3)])
    else:
        cfg = B.make_cfg(width=48, loop=(0, 1, 1), layers=[
            B.retention(heads=1, dim=48, vdim=48, rot_dims=2, decay=[1.0]),
            B.parallel(heads=1, kv_heads=1, dim=48, vdim=48, window=2, conv=1, scale=1.0, bias_max=3, rows=2, inner=48, state=1, dt_rank=1, conv2=1, mlp=B.dense(1))])
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
    """Prefill against token-by-token decoding, portions down to two tokens, unequal requests batched, a long decode tail that a
    window passes over, blocks and state slots that are freed and taken again (12 blocks of 16 where the four requests need 22; four
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
def test_a_far_token_decides_after_hundreds_of_steps(dtype):
    """A sequence of 600 tokens whose last logits still hang on the first tokens through slowly forgetting recurrences (decays of 1
    in the retention, small step sizes in the scan); whole prompt, portions that cut pages and chunks, and decoding agree with the
    oracle.  In bf16 the prompt takes the chunk kernels."""
    cfg = B.make_cfg(width=64, vocab=90, loop=(0, 1, 2), layers=[B.retention(heads=2, dim=32, vdim=32, rot_dims=8, decay=[1.0, 0.999]),
                                                                 B.parallel(heads=2, kv_heads=1, dim=16, vdim=16, inner=48, state=8, window=20)])
    w = B.make_weights(cfg, 12)
    w["l1.mix.right.dt.b"] = torch.full((48,), -6.0)
    w["l1.mix.right.A_log"] = torch.full((48, 8), -2.0)
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
    r = B.make_runner(cfg, w, "float32")
    assert r.cfg.n_layers == 6 and len(r.run_layers) == 6
    looped = sum(t.numel() for t in r._weights)
    once = B.make_runner(B.make_cfg(loop=None), {k: v for k, v in w.items() if k != "loop.step"}, "float32")
    assert looped == sum(t.numel() for t in once._weights) + 2 * cfg["width"]
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
    """Sizes that take the tensor-core kernels: steps that carry portions of many rows (chunks), of a few rows and single decoded
    tokens of different sequences; every request gets what it gets alone, and the oracle's logits within bf16 noise."""
    cfg = B.make_cfg(width=128, vocab=150, loop=(0, 1, 2), layers=[
        B.retention(heads=2, dim=64, vdim=48, rot_dims=32, decay=[0.999, 0.9]),
        B.parallel(heads=4, kv_heads=2, dim=32, vdim=32, window=50, conv=3, inner=128, state=16, dt_rank=8, conv2=4, mlp=B.dense(128))])
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
        assert np.median(e) < 0.02 and (e < 0.08).mean() > 0.95, (n, float(np.median(e)), float(e.max()))
        assert np.median(d) < 0.02 and (d < 0.08).mean() > 0.95, (n, float(np.median(d)), float(d.max()))
    assert len(eng.blocks.free) == 12
    r.close()


def test_greedy_generation_through_the_engines_own_scheduler(model_a, tmp_path):
    """A checkpoint directory goes through the registry, the weight loader, LLMEngine.generate and the scheduler (which hands out
    blocks and state slots and overlaps steps); prompts of unequal length decode side by side."""
    cfg, w = model_a
    path = str(tmp_path / "ckpt")
    U.write_checkpoint(path, cfg, w)
    pc = pkg("config").load_model_config(path)
    assert type(pc).__name__ == "BofusunConfig"
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
    p = _prompt(cfg, 19, 31)
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
