"""The Kulesun decoder through the framework against the plain implementation (tests/plain_kulesun.py): each
mechanism alone, whole prompts layer by layer, portions, decoding, unequal batches, reuse of slots and pages, far keys
and page borders made to stand out, the first tokens, other sizes, the entry point, the replay program."""
import math
import os

import pytest
import torch

import plain_kulesun as plain
from helpers import random_tokens, read_folder, rel_err
from kulesun_cases import (CASES, attn, draw_case, latent, layer, make_folder, model, plain_logits, rot, rounded_logits,
                           write_case)
from test_gpu_felolorn import close, load, run_cut

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
PS = 64


def _K():
    from gogguf_b200.csrc import kernels
    return kernels


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def _batch(lens):
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    return _i32(cu), _i32([b for b, n in enumerate(lens) for _ in range(n)])


def _gen(seed):
    return torch.Generator().manual_seed(seed)


# ----------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("N,K", [(456, 264), (1000, 512), (2056, 1024), (20, 80), (137, 64)])
def test_bias_inside_the_products(N, K):
    """Every form of the product: decode (with and without a K split), prompts of several lengths, adding into float32
    rows with and without row statistics, a folded norm, the plain kernel."""
    from gogguf_b200.parts.base import Linear, RowStats, Runtime, Workspace
    g = _gen(N + K)
    w, b = torch.randn(N, K, generator=g) * 0.1, torch.randn(N, generator=g)
    for dt in (torch.bfloat16, torch.float32):
        rt = Runtime(dtype=dt, device=torch.device(DEV))
        ws = Workspace(rt.device)
        wd = w.to(dt)
        lin = Linear(wd, rt, bias=b)
        for m in (1, 7, 33, 100, 128, 129, 300, 700):
            x = torch.randn(m, K, generator=g).to(dt)
            want = x.double() @ wd.double().t() + b.double()
            tol = 3e-6 if dt == torch.float32 else 6e-3
            out = torch.empty(m, N, dtype=dt, device=DEV)
            lin(x.to(DEV), out, ws=ws)
            assert rel_err(out, want) < tol, (m, dt)
            res = torch.randn(m, N, generator=g)
            acc = res.to(DEV)
            lin(x.to(DEV), acc, accumulate=True, ws=ws)
            assert rel_err(acc, res.double() + want) < 3e-5, (m, dt, "added")
            if dt == torch.bfloat16 and N % 8 == 0 and lin.tensor_core:
                acc = res.to(DEV)
                st = RowStats(torch.empty(m, N, dtype=torch.bfloat16, device=DEV), torch.empty(m, (N + 127) // 128, device=DEV))
                lin(x.to(DEV), acc, accumulate=True, ws=ws, emit=st)
                assert st.fresh and rel_err(acc, res.double() + want) < 3e-5 and rel_err(st.xhat, acc.double()) < 6e-3
                assert rel_err(st.ssq.sum(-1), (acc.double() ** 2).sum(-1).cpu()) < 1e-5
    # a folded norm: the factor multiplies the sums, the bias is added after it
    rt = Runtime(dtype=torch.bfloat16, device=torch.device(DEV))
    lin = Linear(w.to(torch.bfloat16), rt, bias=b)
    nw = 1.0 + torch.randn(K, generator=g) * 0.1
    lin.fold_input_norm(nw, 1e-5)
    for m in (3, 60, 200, 600):
        x = torch.randn(m, K, generator=g) * 5
        want = plain.rms_unit(x.double(), 1e-5) @ lin.weight.double().cpu().t() + b.double()
        st = RowStats(torch.empty(m, K, dtype=torch.bfloat16, device=DEV), torch.empty(m, (K + 127) // 128, device=DEV))
        out = torch.empty(m, N, dtype=torch.float32, device=DEV)
        lin(st.ensure(x.to(DEV)), out, ws=Workspace(rt.device))
        assert rel_err(out, want) < 6e-3, m


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("G,d,dv,unit", [(2, 12, 20, True), (1, 64, 128, True), (5, 8, 40, False), (3, 128, 64, True)])
def test_keys_and_values_into_the_cache(dt, G, d, dv, unit):
    """Values normed over each head, the first layer's kept, a later layer's mixed with them, the cache's rows where the
    page table says; a padding row writes nothing."""
    K = _K()
    g = _gen(G * dv)
    lens, starts = (70, 1, 5), (0, 63, 130)
    T, pad = sum(lens), 16
    row = torch.randn(T, pad + G * (d + dv) + 8, generator=g).to(dt)
    cu, sot = _batch(lens)
    pos = [s + i for s, n in zip(starts, lens) for i in range(n)]
    table = torch.randperm(9, generator=g).reshape(3, 3)
    sot[T - 1] = -1
    first = torch.randn(T, G * dv, generator=g)
    v = row[:, pad + G * d:pad + G * (d + dv)].double().reshape(T, G, dv)
    own = plain.rms_unit(v, 1e-4) if unit else v
    mixed = plain.mixed_values(own, first.double().reshape(T, G, dv), 0.3)
    tol = 1e-6 if dt == torch.float32 else 6e-3
    for mode in ("alone", "keep", "mix"):
        kp = torch.full((9, G, PS, d), 7.0, dtype=dt, device=DEV)
        vp = torch.full((9, G, PS, dv), 7.0, dtype=dt, device=DEV)
        keep = torch.full((T, G * dv), 9.0, device=DEV)
        K.head_kv_prep(row.to(DEV), pad, pad + G * d, kp, vp, _i32(pos), sot, _i32(table.tolist()), PS, T, G, d, dv, unit, 1e-4,
                       first.to(DEV) if mode == "mix" else None, 0.3, keep if mode == "keep" else None)
        want = mixed if mode == "mix" else own
        seen = torch.zeros(9, PS, dtype=torch.bool)
        for t in range(T - 1):
            pg, sl = int(table[int(sot[t]), pos[t] // PS]), pos[t] % PS
            seen[pg, sl] = True
            assert torch.equal(kp[pg, :, sl].cpu().reshape(-1), row[t, pad:pad + G * d])
            assert rel_err(vp[pg, :, sl], want[t]) < tol, (mode, t)
        assert float((kp.float().cpu().permute(0, 2, 1, 3)[~seen] - 7.0).abs().max()) == 0.0
        assert float((vp.float().cpu().permute(0, 2, 1, 3)[~seen] - 7.0).abs().max()) == 0.0
        if mode == "keep":
            assert rel_err(keep[:T - 1], own[:T - 1].reshape(T - 1, -1)) < 1e-5 and float(keep[T - 1].min()) == 9.0


def _mixed_reference(q, k, v, gate, talk, pos, lens, scale, cap, coef, every, one, window=0):
    """q [T, H, d] of the step's tokens, k [b][n, G, d] and v [b][n, G, dv] everything each sequence has cached."""
    out = []
    t = 0
    H = q.shape[1]
    for b, n in enumerate(lens):
        G = k[b].shape[1]
        own = [h // (H // G) for h in range(H)]
        for _ in range(n):
            p = int(pos[t])
            tau = plain.query_temperature(p + 1, coef, every)[p] if coef else 1.0
            s = plain.bounded(torch.einsum("hd,jhd->hj", q[t] * tau, k[b][:p + 1][:, own]) * scale, cap)
            if window:
                s[:, :max(0, p - window + 1)] = -math.inf
            a = plain.weights_with_one(s) if one else torch.softmax(s, dim=-1)
            a = torch.einsum("hg,gj->hj", talk, a)
            o = torch.einsum("hj,jhe->he", a, v[b][:p + 1][:, own])
            out.append(o * plain.sigmoid(gate[t])[:, None] if gate is not None else o)
            t += 1
    return torch.stack(out)


def _prompt_form(K, row, g_off, kf, vf, talk, pos, lens, sot, cu, table, H, G, d, dv, scale, want, nv, kw, tol=1.2e-2):
    """The tcgen05 form on a step of stretches `lens` against the wanted rows."""
    T, ends = len(pos), []
    for n in lens:
        ends.append(pos[sum(lens[:len(ends) + 1]) - 1] + 1)
    o = torch.empty(T, H * dv, dtype=torch.bfloat16, device=DEV)
    u = torch.full((T * H * G * dv,), 1e30, device=DEV)
    ml = torch.full((T * H * 2,), 1e30, device=DEV)
    K.mixed_head_attention_prompt(row.to(DEV), g_off, kf.to(DEV), vf.to(DEV), o, talk.to(DEV), sot, cu, _i32(ends), table, PS, T,
                                  len(lens), H, G, d, dv, scale, u, ml, value_heads=nv, **kw)
    from gogguf_b200.csrc.tcgen05_gemm import check_status
    check_status(torch.device(DEV))
    assert rel_err(o, want) < tol, ("prompt form", lens, nv, rel_err(o, want))


@pytest.mark.parametrize("cap,factor", [(0.0, 1.0), (0.0, 30.0), (60.0, 12.0), (30.0, 1.0), (30.0, 25.0), (2.0, 3.0)])
def test_prompt_form_with_scores_of_every_size(cap, factor):
    """Small and large scores: bounds that serve as their own reference and bounds that are too wide for it, no bound,
    maxima that grow from page to page, scores beyond the polynomial's range."""
    K = _K()
    H, G, d, dv, n = 4, 2, 64, 128, 300
    g = _gen(int(cap * 10 + factor))
    kf = torch.randn(5, G, PS, d, generator=g)
    kf = (kf * torch.linspace(0.2, 1.5, 5).reshape(5, 1, 1, 1)).to(torch.bfloat16)      # later pages score higher
    vf = torch.randn(5, G, PS, dv, generator=g).to(torch.bfloat16)
    row = torch.randn(n, H * d + 8, generator=g).to(torch.bfloat16)
    talk = torch.eye(H) + torch.randn(H, H, generator=g) / H
    ks, vs = (torch.cat([f[p].permute(1, 0, 2) for p in range(5)]).double() for f in (kf, vf))
    pos = list(range(n))
    kw = dict(cap=cap, coef=0.2, every=30.0, one=True)
    scale = factor / math.sqrt(d)
    want = _mixed_reference(row[:, :H * d].double().reshape(n, H, d), [ks], [vs], row[:, H * d:H * d + H].double(), talk.double(), pos,
                            [n], scale, cap, 0.2, 30.0, True).reshape(n, H * dv)
    cu, sot = _batch((n,))
    for nv in (1, 2):
        _prompt_form(K, row, H * d, kf, vf, talk, pos, [n], sot, cu, _i32([list(range(5))]), H, G, d, dv, scale, want, nv, kw)


@pytest.mark.parametrize("H,G,d,dv,cap,temp,one,gated", [
    (8, 4, 64, 64, 18.0, (0.25, 16.0), True, True), (6, 2, 12, 20, 5.0, (0.5, 7.0), True, True),
    (8, 1, 32, 128, 0.0, None, True, True), (3, 3, 128, 40, 10.0, (1.0, 1.0), True, False),
    (5, 1, 40, 32, 30.0, (-0.1, 3.0), False, True), (12, 4, 64, 96, 15.0, None, True, True),
    (32, 8, 128, 128, 25.0, (0.1, 64.0), True, True), (1, 1, 16, 16, 3.0, None, True, True), (24, 1, 8, 8, 0.0, (0.2, 9.0), True, True)])
def test_attention_with_mixed_heads_alone(H, G, d, dv, cap, temp, one, gated):
    """The plain kernel in float32 and in bfloat16 and the tensor-core kernel against the sums written out: prompts of
    unequal lengths, portions that go on from the cache, one token each; pages in no particular order; shares of the
    keys; tiles of few rows; a padding row."""
    K = _K()
    g = _gen(H * d + dv)
    n_pages = 24
    coef, every = temp or (0.0, 1.0)
    scale = 1.3 / math.sqrt(d)
    talk = torch.eye(H) + torch.randn(H, H, generator=g) / H
    perm = torch.randperm(n_pages, generator=g).tolist()
    table = _i32([perm[0:8], perm[8:16], perm[16:24]])
    kf = torch.randn(n_pages, G, PS, d, generator=g).to(torch.bfloat16)
    vf = torch.randn(n_pages, G, PS, dv, generator=g).to(torch.bfloat16)
    seq = lambda pool, b: torch.cat([pool[p].permute(1, 0, 2) for p in table[b].tolist()]).double()
    ks, vs = [seq(kf, b) for b in range(3)], [seq(vf, b) for b in range(3)]
    done = [0, 0, 0]
    g_off = H * d + 8 if gated else -1
    width = H * d + 8 + (H + 7) // 8 * 8
    window = {12: 70, 3: 100}.get(H, 0)
    kw = dict(cap=cap, coef=coef, every=every, one=one, window=window)
    for lens in ((130, 1, 67), (65, 180, 2), (1, 1, 1), (2, 1, 3), (1, 1, 1)):
        cu, sot = _batch(lens)
        T = sum(lens)
        pos = [done[b] + i for b, n in enumerate(lens) for i in range(n)]
        row = torch.randn(T, width, generator=g).to(torch.bfloat16)
        want = _mixed_reference(row[:, :H * d].double().reshape(T, H, d), ks, vs,
                                row[:, g_off:g_off + H].double() if gated else None, talk.double(), pos, lens, scale, cap, coef,
                                every, one, window).reshape(T, H * dv)
        for dt in (torch.float32, torch.bfloat16):
            o = torch.empty(T, H * dv, dtype=dt, device=DEV)
            K.mixed_head_attention_plain(row.to(dt).to(DEV), g_off, kf.to(dt).to(DEV), vf.to(dt).to(DEV), o, talk.to(DEV), _i32(pos),
                                         sot, table, PS, T, H, G, d, dv, scale, **kw)
            assert rel_err(o, want) < (2e-5 if dt == torch.float32 else 6e-3), (lens, dt)
        if not K.mixed_head_mma_takes(H, G, d, dv, PS):
            assert d % 8 or dv % 8
        else:
            forms = [(1, 0), (3, 0)] + ([(1, max(lens)), (3, max(lens)), (7, max(lens))] if max(lens) <= 3 else [])
            for ns, mx in forms:
                o = torch.empty(T, H * dv, dtype=torch.bfloat16, device=DEV)
                u = torch.full((T * H * ns * G * dv,), 1e30, device=DEV)
                ml = torch.full((T * H * ns * 2,), 1e30, device=DEV)
                K.mixed_head_attention_mma(row.to(DEV), g_off, kf.to(DEV), vf.to(DEV), o, talk.to(DEV), _i32(pos), sot, cu, table,
                                           PS, T, 3, H, G, d, dv, scale, u, ml, nsplit=ns, max_new=mx, **kw)
                assert rel_err(o, want) < 1.2e-2, (lens, ns, mx, rel_err(o, want))
            if max(lens) <= 3 and K.mixed_head_decode_takes(H, G, d, dv, PS):
                for ns in (1, 3, 8):
                    o = torch.empty(T, H * dv, dtype=torch.bfloat16, device=DEV)
                    scores = torch.full((T, H, 8 * PS), 1e30, device=DEV)
                    ml, part = torch.full((T * H * ns * 2,), 1e30, device=DEV), torch.full((T * H * ns * dv,), 1e30, device=DEV)
                    K.mixed_head_attention_decode(row.to(DEV), g_off, kf.to(DEV), vf.to(DEV), o, talk.to(DEV), _i32(pos), sot, table, PS,
                                                  T, H, G, d, dv, scale, scores, ml, part, ns, **kw)
                    assert rel_err(o, want) < 6e-3, (lens, ns, rel_err(o, want))
            for nv in (1, 2) + ((4,) if dv <= 64 else ()):
                _prompt_form(K, row, g_off, kf, vf, talk, pos, lens, sot, cu, table, H, G, d, dv, scale, want, nv, kw)
        done = [x + n for x, n in zip(done, lens)]
    cu, sot = _batch((1, 1))
    sot[1] = -1
    for which in ("plain", "mma", "decode"):
        o = torch.full((2, H * dv), 5.0, dtype=torch.bfloat16, device=DEV)
        row = torch.randn(2, width, generator=g).to(torch.bfloat16).to(DEV)
        args = (row, g_off, kf.to(DEV), vf.to(DEV), o, talk.to(DEV), _i32([done[0], 0]), sot)
        if which == "plain":
            K.mixed_head_attention_plain(*args, table[:2].contiguous(), PS, 2, H, G, d, dv, scale, **kw)
        elif which == "decode" and K.mixed_head_decode_takes(H, G, d, dv, PS):
            K.mixed_head_attention_decode(*args, table[:2].contiguous(), PS, 2, H, G, d, dv, scale, torch.empty(2, H, 8 * PS, device=DEV),
                                          torch.empty(4 * H, device=DEV), torch.empty(2 * H * dv, device=DEV), 1, **kw)
        elif which == "mma" and K.mixed_head_mma_takes(H, G, d, dv, PS):
            K.mixed_head_attention_mma(*args, cu, table[:2].contiguous(), PS, 2, 2, H, G, d, dv, scale,
                                       torch.empty(2 * H * G * dv, device=DEV), torch.empty(4 * H, device=DEV), max_new=1, **kw)
        else:
            continue
        assert float(o[1].float().abs().max()) == 0.0 and float(o[0].float().abs().max()) > 0.0


def test_scores_that_are_all_far_below_the_one():
    """Every score is far below zero, so the one in the denominator takes nearly everything: outputs of 1e-6 keep their
    digits, with and without shares of the keys."""
    K = _K()
    H, G, d, dv, n = 2, 1, 64, 64, 200
    g = _gen(9)
    q = torch.zeros(1, H * d + 8)
    q[0, 0] = q[0, d] = 4.0
    kf = torch.zeros(4, G, PS, d)
    kf[..., 0] = -4.0
    vf = torch.randn(4, G, PS, dv, generator=g)
    want = _mixed_reference(q[:, :H * d].double().reshape(1, H, d), [torch.cat([kf[p].permute(1, 0, 2) for p in range(4)]).double()],
                            [torch.cat([vf[p].to(torch.bfloat16).permute(1, 0, 2) for p in range(4)]).double()], None, torch.eye(H).double(),
                            [n - 1], [1], 1.0, 0.0, 0.0, 1.0, True).reshape(1, -1)
    cu, sot = _batch((1,))
    for ns in (1, 2, 4):
        o = torch.empty(1, H * dv, dtype=torch.bfloat16, device=DEV)
        K.mixed_head_attention_mma(q.to(torch.bfloat16).to(DEV), -1, kf.to(torch.bfloat16).to(DEV), vf.to(torch.bfloat16).to(DEV), o,
                                   torch.eye(H, device=DEV), _i32([n - 1]), sot, cu, _i32([[0, 1, 2, 3]]), PS, 1, 1, H, G, d, dv, 1.0,
                                   torch.empty(H * ns * dv, device=DEV), torch.empty(H * ns * 2, device=DEV), one=True, nsplit=ns,
                                   max_new=1)
        assert 0 < float(want.abs().max()) < 1e-4 and rel_err(o, want) < 1.2e-2
        K.mixed_head_attention_decode(q.to(torch.bfloat16).to(DEV), -1, kf.to(torch.bfloat16).to(DEV), vf.to(torch.bfloat16).to(DEV), o,
                                      torch.eye(H, device=DEV), _i32([n - 1]), sot, _i32([[0, 1, 2, 3]]), PS, 1, H, G, d, dv, 1.0,
                                      torch.empty(1, H, 256, device=DEV), torch.empty(H * ns * 2, device=DEV),
                                      torch.empty(H * ns * dv, device=DEV), ns, one=True)
        assert rel_err(o, want) < 6e-3


@pytest.mark.parametrize("dt,qdt", [(torch.float32, torch.float32), (torch.bfloat16, torch.float32), (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("H,d,r,R,dims,pairing", [(3, 20, 6, 28, 6, "halves"), (4, 64, 32, 128, 32, "halves"), (2, 16, 12, 16, 4, "halves"),
                                                  (4, 8, 16, 64, 16, "adjacent")])
def test_rotation_of_the_latent_layers_parts(dt, qdt, H, d, r, R, dims, pairing):
    """Both pairings, whole and partial rotations; the latent's norm; the cache row and its dense copy."""
    from plain_dinuzen import rotate_adjacent
    K = _K()
    g = _gen(H + R)
    T = 70
    rt = dict(dims=dims, base=900.0, scaling=dict(factor=2.0, original=64, fast=16.0, slow=1.0))
    f, mag = plain.yarn_frequencies(rt)
    ang = torch.arange(T, dtype=torch.float64)[:, None] * f[None]
    cos, sin = (torch.cos(ang) * mag).float().to(DEV), (torch.sin(ang) * mag).float().to(DEV)
    x = torch.randn(T, H * (d + r) + R + r + 8, generator=g).to(dt)
    nw = torch.randn(R, generator=g)
    pool = torch.zeros(2, PS, R + r + 2, dtype=dt, device=DEV)
    dense = torch.empty(T, R + r, dtype=dt, device=DEV)
    qcat = torch.zeros(T, H, R + r, dtype=qdt, device=DEV)
    xd = x.to(DEV)
    cu, sot = _batch((T,))
    K.latent_prep(xd[:, :H * (d + r)], xd[:, H * (d + r):H * (d + r) + R + r], nw.to(DEV), 1e-5, cos, sin, dims, _i32(list(range(T))), sot,
                  _i32([[1, 0]]), PS, pool, qcat, T, H, d, r, R, dense=dense, pairing=pairing)
    turn = plain.rotate_halves if pairing == "halves" else rotate_adjacent
    q = x[:, :H * (d + r)].double().reshape(T, H, d + r)[..., d:]
    dkv = x[:, H * (d + r):H * (d + r) + R + r].double()
    row = torch.cat([plain.rms_unit(dkv[:, :R], 1e-5) * nw.double(), turn(dkv[:, R:], rt)], dim=1)
    assert rel_err(qcat[:, :, R:], turn(q, rt)) < (3e-6 if qdt == torch.float32 else 6e-3)
    assert rel_err(dense, row) < (3e-6 if dt == torch.float32 else 6e-3)
    got = torch.cat([pool[1], pool[0]])[:T]
    assert torch.equal(got[:, :R + r], dense) and float(got[:, R + r:].float().abs().max()) == 0.0


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_per_head_products_behind_a_gate(dt):
    from gogguf_b200.csrc import fast_latent
    K = _K()
    g = _gen(4)
    for T, H, N, R in ((5, 3, 24, 32), (130, 4, 72, 64), (1, 2, 20, 48)):
        x, w = torch.randn(T, H, R, generator=g).to(dt), (torch.randn(H, N, R, generator=g) * 0.2).to(dt)
        wide = torch.randn(T, 16 + H * N, generator=g).to(dt)
        want = torch.einsum("thr,hnr->thn", x.double(), w.double()) * 0.7
        want = want.reshape(T, H * N) * plain.sigmoid(wide[:, 16:].double())
        forms = [K.headwise_gemm] + ([fast_latent.headwise_gemm_mma] if dt == torch.bfloat16 else [])
        for fn in forms:
            out = torch.empty(T, H * N, dtype=dt, device=DEV)
            fn(x.to(DEV), H * R, R, w.to(DEV), out, H * N, N, T, 0.7, gate=wide.to(DEV)[:, 16:])
            assert rel_err(out, want) < (2e-6 if dt == torch.float32 else 6e-3), (T, fn.__name__)


def test_factor_on_the_logits_with_and_without_a_bound():
    K = _K()
    z = torch.randn(5, 33, generator=_gen(2)) * 20
    for cap, f in ((0.0, 0.3), (10.0, 2.0), (10.0, 1.0)):
        zd = z.to(DEV)
        K.softcap(zd, cap, scale=f)
        assert rel_err(zd, plain.bounded(z.double() * f, cap)) < 2e-6


def _one_layer(mixer, ff=None, width=64, vocab=61, eps=1e-5):
    return model(vocab, width, eps, [layer(mixer, ff)], 2.0, 0.5)


ALONE = {
    "mixed_heads": _one_layer(attn(6, 2, 12, 20, 0.3, 15.0, (0.5, 7.0))),
    "mixed_heads_wide": _one_layer(attn(8, 2, 64, 128, 0.125, 20.0, (0.2, 30.0)), width=128),
    "mixed_heads_plain_scores": _one_layer(attn(2, 2, 8, 8, 0.35, None, None, v_mix=False)),
    "mixed_heads_long": _one_layer(attn(3, 1, 136, 264, 0.1, 12.0, (0.1, 2.0))),
    "latent": _one_layer(latent(3, 20, 6, 12, 28, 0.25, rot(6, 10000.0, (4.0, 64, 16.0, 2.0)))),
    "latent_wide": _one_layer(latent(4, 64, 32, 64, 128, 0.1, rot(32, 500.0, (8.0, 32, 8.0, 1.0))), width=128),
    "latent_unstretched": _one_layer(latent(2, 32, 16, 96, 48, 0.2, rot(16, 1e5))),
    "dense": _one_layer(attn(1, 1, 8, 8, 0.3), 100),
    "dense_wide": _one_layer(attn(1, 1, 8, 8, 0.3), 320, width=128),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_one_mechanism_in_a_layer_of_its_own(tmp_path_factory, name, dtype):
    """A model of one layer: its mixer (or feed-forward) decides the layer's output.  Whole, cut, token by token."""
    folder = write_case(tmp_path_factory.getbasetemp(), "alone_" + name, ALONE[name], 17, dtype, std=0.2)
    cfg, w = read_folder(folder)
    tokens = random_tokens(cfg["vocab"], 140, seed=3)
    layers, layers32 = [], []
    want = plain_logits(cfg, w, tokens, layers)
    own32 = plain_logits(cfg, w, tokens, layers32, torch.float32)
    from gogguf_b200.engine import LayerTaps, StepEntry
    m, cache, st = load(folder, dtype)
    got_layers = []
    slot = cache.open()
    got = st.step([StepEntry(slot, tokens, want=list(range(len(tokens))))],
                  LayerTaps(on_layer=lambda i, rows: got_layers.append(rows.clone()))).clone()
    cache.close(slot)
    assert close(got_layers[0], layers[0], dtype, own32=layers32[0]), (rel_err(got_layers[0], layers[0]), name)
    assert close(got, want, dtype, own32=own32), (rel_err(got, want), name)
    for cuts in ([64, 2, 70], [1, 63, 1, 65], []):
        out = run_cut(st, cache, tokens if cuts else tokens[:70], cuts)
        ref = want if cuts else want[:70]
        assert close(out, ref, dtype, own32=own32[:ref.shape[0]], gauge=got[:ref.shape[0]]), (rel_err(out, ref), name, cuts)


def test_attention_with_its_options_left_out(tmp_path_factory):
    """Another design's use of the mixer: no biases, no mixing of heads, no gate, no one in the denominator, values as they
    are.  The same tensors with the identity, zeros and closed options through the plain functions."""
    from gogguf_b200.config.spec import BlockSpec, PartSpec
    from gogguf_b200.engine import Model, StepEntry, Stepper
    import dataclasses
    folder = make_folder(tmp_path_factory.getbasetemp(), "S", "float32")
    cfg, w = read_folder(folder)
    from gogguf_b200.config import config_from_dict
    spec = config_from_dict(cfg).to_spec()
    blocks, drop = [], []
    for i, b in enumerate(spec.blocks):
        ps = b.parts["mixer"]
        if ps.kind == "mixed_head_attention":
            off = dict(bias=False, talking=False, head_gate=False, extra_one=False, unit_values=False, value_mix=None)
            b = BlockSpec(b.arrangement, {**b.parts, "mixer": PartSpec(kind=ps.kind, prefix=ps.prefix, params={**ps.params, **off})})
            drop += [ps.prefix + n for n in ("q.b", "k.b", "v.b", "o.b", "talk", "g", "vmix")]
        blocks.append(b)
    spec = dataclasses.replace(spec, blocks=tuple(blocks))
    tensors = {n: t for n, t in w.items() if n not in drop}
    tokens = random_tokens(cfg["vocab"], 90, seed=2)
    eps = cfg["norm"]["eps"]

    def bare(m, p, h):
        n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        q, k, v = (plain.linear(h, w, p + x) for x in "qkv")
        qt = m.get("q_temp")
        tau = plain.query_temperature(n, qt["coef"], qt["every"]) if qt else torch.ones(n, dtype=torch.float64)
        own = [x // (H // G) for x in range(H)]
        s = torch.einsum("ihd,jhd->hij", q.reshape(n, H, d) * tau[:, None, None], k.reshape(n, G, d)[:, own]) * m["scale"]
        a = torch.softmax(plain.bounded(s, m.get("softcap") or 0.0) + plain.unseen(n, h.dtype), dim=-1)
        return plain.linear(torch.einsum("hij,jhe->ihe", a, v.reshape(n, G, dv)[:, own]).reshape(n, H * dv), w, p + "o")

    E = w["embed"].double()
    x = E[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = plain.norm_about_one(x, w[p + "norm1"], eps)
        y = (bare(l["mixer"], p + "mix.", h) if l["type"] == "attention" else plain.latent_attention(l["mixer"], w, p + "mix.", h, eps))
        x = x + plain.norm_about_one(y, w[p + "norm1b"], eps)
        if l["mlp"] is not None:
            y = plain.feed_forward(w, p + "mlp.", plain.norm_about_one(x, w[p + "norm2"], eps))
            x = x + plain.norm_about_one(y, w[p + "norm2b"], eps)
    want = plain.norm_about_one(x, w["final.norm"], eps) @ E.t() * cfg["logit_scale"]
    for dtype in ("float32", "bfloat16"):
        m = Model(spec, tensors, dtype=dtype)
        cache = m.new_cache(max_tokens=512)
        for cuts in ([90], [64, 2]):
            got = run_cut(Stepper(m, cache), cache, tokens, cuts)
            assert rel_err(got, want) < (1e-4 if dtype == "float32" else 1e-1), (dtype, cuts, rel_err(got, want))


# ----------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("name", ["S", "ONE", "W"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts_and_every_layer(tmp_path_factory, name, dtype):
    from gogguf_b200.engine import LayerTaps, StepEntry
    folder = make_folder(tmp_path_factory.getbasetemp(), name, dtype)
    cfg, w = read_folder(folder)
    m, cache, st = load(folder, dtype)
    for n in (1, 2, 3, 150):
        tokens = random_tokens(cfg["vocab"], n, seed=n)
        want_layers, layers32 = [], []
        want = plain_logits(cfg, w, tokens, want_layers)
        logits32 = plain_logits(cfg, w, tokens, layers32, torch.float32)
        got_layers = []
        slot = cache.open()
        got = st.step([StepEntry(slot, tokens, want=list(range(n)))],
                      LayerTaps(on_layer=lambda i, rows: got_layers.append(rows.clone()))).clone()
        cache.close(slot)
        assert len(got_layers) == len(cfg["layers"])
        for i, (a, b) in enumerate(zip(got_layers, want_layers)):
            assert close(a, b, dtype, own32=layers32[i]), (rel_err(a, b), name, n, "layer", i)
        assert close(got, want, dtype, own32=logits32), (rel_err(got, want), name, n)
    if dtype == "bfloat16":
        # the plain kernels on the same weights are the twins of the tensor-core kernels
        _, cache2, st2 = load(folder, dtype, fast=False)
        assert close(run_cut(st2, cache2, tokens, [len(tokens)]), want, dtype)


def test_which_kernels_the_wide_model_takes(tmp_path_factory):
    folder = make_folder(tmp_path_factory.getbasetemp(), "W", "bfloat16")
    m, _, _ = load(folder, "bfloat16")
    K = _K()
    for b in m.blocks:
        assert b.mixer_folded and (b.feed_forward is None or b.ff_folded)
        x = b.mixer
        if hasattr(x, "talk"):
            assert x._mma and K.mixed_head_mma_takes(x.H, x.G, x.d, x.dv, PS)
        else:
            assert x._fast is not None and x.kv_up is not None and x.pairing == "halves"


@pytest.mark.parametrize("name,dtype", [("S", "float32"), ("S", "bfloat16"), ("ONE", "float32"), ("W", "float32"),
                                        ("W", "bfloat16")])
def test_portions_and_decoding_equal_the_whole_prompt(tmp_path_factory, name, dtype):
    folder = make_folder(tmp_path_factory.getbasetemp(), name, dtype)
    cfg, w = read_folder(folder)
    tokens = random_tokens(cfg["vocab"], 171, seed=12)
    want = plain_logits(cfg, w, tokens)
    own32 = plain_logits(cfg, w, tokens, None, torch.float32)
    m, cache, st = load(folder, dtype)
    whole = None
    for cuts in ([171], [64, 64, 43], [2, 2, 61, 3, 100], [63, 2, 70], [130], [1, 65, 2, 2], [1, 129, 41], [1, 1, 1, 3, 160]):
        got = run_cut(st, cache, tokens, cuts)
        assert close(got, want, dtype, own32=own32, gauge=whole), (rel_err(got, want), name, cuts)
        whole = got if whole is None else whole
    # token by token from the first one, through captured graphs
    _, cache_g, st_g = load(folder, dtype, graphs=True)
    got = run_cut(st_g, cache_g, tokens[:90], [])
    assert close(got, want[:90], dtype, own32=own32[:90], gauge=whole[:90]), rel_err(got, want[:90])
    assert st_g.replays >= 89


@pytest.mark.parametrize("name,dtype", [("S", "float32"), ("S", "bfloat16"), ("W", "bfloat16"), ("ONE", "float32")])
def test_unequal_batches_and_reused_slots_and_pages(tmp_path_factory, name, dtype):
    """Requests of different lengths in one batch, decoded together while the short ones leave; the slots and pages they
    give back are taken by the next batch (the cache is sized so that it must)."""
    from gogguf_b200.engine import StepEntry
    folder = make_folder(tmp_path_factory.getbasetemp(), name, dtype)
    cfg, w = read_folder(folder)
    m, cache, st = load(folder, dtype, max_tokens=448, graphs=True)
    got_rows, want_rows, own_rows = [], [], []
    for wave in range(3):
        reqs = [random_tokens(cfg["vocab"], n, seed=100 * wave + n) for n in (1, 65, 130, 7)]
        tails = [3, 20, 9, 40]
        full = [r + random_tokens(cfg["vocab"], t, seed=7 + t + wave) for r, t in zip(reqs, tails)]
        oracle = [plain_logits(cfg, w, f) for f in full]
        own = [plain_logits(cfg, w, f, None, torch.float32) for f in full]
        slots = [cache.open() for _ in reqs]
        out = st.step([StepEntry(s, r, want=[len(r) - 1]) for s, r in zip(slots, reqs)]).clone()
        for i, r in enumerate(reqs):
            got_rows.append(out[i]); want_rows.append(oracle[i][len(r) - 1]); own_rows.append(own[i][len(r) - 1])
        live = list(range(len(reqs)))
        for k in range(max(tails)):
            live = [i for i in live if k < tails[i]]
            out = st.step([StepEntry(slots[i], [full[i][len(reqs[i]) + k]], want=[0]) for i in live]).clone()
            for j, i in enumerate(live):
                got_rows.append(out[j]); want_rows.append(oracle[i][len(reqs[i]) + k])
                own_rows.append(own[i][len(reqs[i]) + k])
            for i in live:
                if k == tails[i] - 1:
                    cache.close(slots[i])
        cache.check()
        assert cache.live_slots == 0
    got, want = torch.stack(got_rows), torch.stack(want_rows)
    assert close(got, want, dtype, own32=torch.stack(own_rows)), rel_err(got, want)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_across_pages(tmp_path_factory, dtype):
    """A short prompt and 300 decoded tokens: the sequence crosses four page borders, the temperature steps on."""
    name = "S" if dtype == "float32" else "W"
    folder = make_folder(tmp_path_factory.getbasetemp(), name, dtype)
    cfg, w = read_folder(folder)
    tokens = random_tokens(cfg["vocab"], 305, seed=77)
    want = plain_logits(cfg, w, tokens)
    own32 = plain_logits(cfg, w, tokens, None, torch.float32)
    m, cache, st = load(folder, dtype, max_tokens=512, graphs=True)
    got = run_cut(st, cache, tokens, [5])
    assert close(got, want, dtype, own32=own32), rel_err(got, want)


# ----------------------------------------------------------------------------------------------- made-up weights
MARKED, ASKING = 1, 5      # token ids: the one that is asked for, the one whose query asks


def _standout_model(tmp, kind, store):
    """A one-layer model without feed-forward whose weights make one token stand out.  The marked token's input has
    a large component along a direction that every other token's input is orthogonal to, the asking token's along
    another.  One key element of every head copies the marked direction, the same element of every query the asking
    direction, and the scale is large: the asking token gives the marked one a score far above all others, wherever it
    lies; every other score lies below the one in the denominator or spreads evenly."""
    from gogguf_b200.weights.loader import write_model_folder
    W, V = 64, 64
    g = _gen(31)
    embed = torch.randn(V, W, generator=g)
    a = embed[MARKED] / embed[MARKED].norm()
    for j in range(V):
        if j != MARKED:
            embed[j] -= (embed[j] @ a) * a
    mdir = embed[ASKING] / embed[ASKING].norm()
    small = lambda *s: torch.randn(*s, generator=g) * 0.02
    mid = lambda *s: torch.randn(*s, generator=g) * 0.3
    p = "l0.mix."
    w = {"embed": embed, "final.norm": torch.zeros(W), "l0.norm1": torch.zeros(W), "l0.norm1b": torch.zeros(W)}
    if kind == "attention":
        H, G, d, dv = 4, 2, 16, 24
        mx = attn(H, G, d, dv, 5.0, 25.0, (0.3, 40.0), v_mix=False)
        q, k = small(H * d, W), small(G * d, W)
        for h in range(H):
            q[h * d + 9] = mdir
        for gg in range(G):
            k[gg * d + 9] = a
        w.update({p + "q": q, p + "k": k, p + "v": mid(G * dv, W), p + "o": mid(W, H * dv), p + "q.b": small(H * d),
                  p + "k.b": small(G * d), p + "v.b": small(G * dv), p + "o.b": small(W), p + "talk": torch.eye(H) + small(H, H),
                  p + "g": mid(H, W)})
    else:
        H, d, r, dv, R = 3, 16, 8, 24, 32
        mx = latent(H, d, r, dv, R, 3.0, rot(r, 10000.0, (2.0, 64, 16.0, 1.0)))
        q, dkv, uk = small(H * (d + r), W), mid(R + r, W), small(H * d, R)
        dkv[3] = 12.0 * a
        dkv[R:] = small(r, W)
        for h in range(H):
            q[h * (d + r) + 6] = mdir
            uk[h * d + 6] = 0.0
            uk[h * d + 6, 3] = 1.0
        w.update({p + "q": q, p + "dkv": dkv, p + "dkv.norm": torch.ones(R), p + "uk": uk, p + "uv": mid(H * dv, R),
                  p + "g": mid(H * dv, W), p + "o": mid(W, H * dv)})
    cfg = model(V, W, 1e-6, [layer(mx, None)], 1.0, 1.0)
    folder = os.path.join(str(tmp), f"standout_{kind}_{store}")
    write_model_folder(folder, cfg, {n: t.to(torch.bfloat16 if store == "bfloat16" else torch.float32) for n, t in w.items()})
    return folder


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_a_token_far_back_at_page_borders_and_at_the_start(tmp_path, dtype, kind):
    """The marked token stands once in a long sequence: first, second, around a page border, hundreds of tokens
    back, just before the end.  The asking token at the end must see it: the same sequence without it gives another row."""
    folder = _standout_model(tmp_path, kind, dtype)
    cfg, w = read_folder(folder)
    m, cache, st = load(folder, dtype)
    n = 330
    for marked in (0, 1, 62, 63, 64, 65, 127, 128, 200, 319, 320, 328):
        tokens = [t if t not in (MARKED, ASKING) else 7 for t in random_tokens(cfg["vocab"], n, seed=marked)]
        tokens[marked], tokens[-1] = MARKED, ASKING
        without = list(tokens)
        without[marked] = 9
        want = plain_logits(cfg, w, tokens)
        moved = rel_err(plain_logits(cfg, w, without)[-1], want[-1])
        assert moved > 0.05, (kind, marked, moved)
        for cuts in ([n], [n - 1], [marked + 1, n - marked - 2], [n - 40]):
            if min(cuts) < 1:
                continue
            got = run_cut(st, cache, tokens, cuts)
            rows = [marked, n - 1]
            assert close(got[rows], want[rows], dtype), (rel_err(got[rows], want[rows]), kind, marked, cuts)


# ----------------------------------------------------------------------------------------------- entry point, others
def test_greedy_generation_through_the_entry_point(tmp_path_factory):
    import gogguf_b200 as gg
    for name, dtype in (("S", "float32"), ("W", "bfloat16")):
        folder = make_folder(tmp_path_factory.getbasetemp(), name, dtype, std=0.3 if dtype == "float32" else None)
        cfg, w = read_folder(folder)
        prompts = [random_tokens(cfg["vocab"], n, 30 + n) for n in (5, 1, 80)]
        engine = gg.load(folder, gg.LoadOptions(dtype=dtype, max_tokens=1024))
        ctx = engine.new_context()
        out = ctx.generate(prompts, gg.GenerateParams(max_tokens=12, stop_token_ids=[], keep_logits=True))
        rows, refs = [], []
        for p, r in zip(prompts, out):
            assert len(r.tokens) == 12 and r.prompt_tokens == len(p) and len(r.logits) == 12
            whole = plain_logits(cfg, w, list(p) + r.tokens[:-1])
            for k, row in enumerate(r.logits):
                assert int(row.argmax()) == r.tokens[k]            # greedy: the token is the best of its own row
                rows.append(row)
                refs.append(whole[len(p) - 1 + k])
        assert close(torch.stack(rows), torch.stack(refs), dtype), rel_err(torch.stack(rows), torch.stack(refs))
        # a second round in the same context reuses the slots and pages the first gave back; without kept logits the
        # loop runs a step ahead of the host and drops the step a finished sequence ran too far
        again = ctx.generate(prompts, gg.GenerateParams(max_tokens=12, stop_token_ids=[]))
        assert [r.tokens for r in again] == [r.tokens for r in out]
        stop = out[2].tokens[4]
        third = ctx.generate(prompts, gg.GenerateParams(max_tokens=12, stop_token_ids=[stop]))
        assert third[2].tokens == out[2].tokens[:out[2].tokens.index(stop)]
        ctx.cache.check()
        assert ctx.cache.live_slots == 0


@pytest.mark.parametrize("seed", list(range(12)))
def test_a_configuration_nobody_chose(tmp_path, seed):
    """Drawn sizes, layer orders and constants; whole, in portions, and a batch of two."""
    from gogguf_b200.engine import StepEntry
    for dtype in ("float32", "bfloat16"):
        cfg = draw_case(seed)
        folder = write_case(tmp_path, f"drawn{seed}", cfg, seed, dtype, std=0.15)
        cfg2, w = read_folder(folder)
        tokens = random_tokens(cfg["vocab"], 97, seed=seed)
        want = plain_logits(cfg2, w, tokens)
        own32 = plain_logits(cfg2, w, tokens, None, torch.float32)
        rounded = rounded_logits(cfg2, w, tokens) if dtype == "bfloat16" else None      # (drawn scores may be large)
        m, cache, st = load(folder, dtype, graphs=True)
        for cuts in ([97], [3, 64, 2, 20], [90]):
            got = run_cut(st, cache, tokens, cuts)
            assert close(got, want, dtype, own32=own32, gauge=rounded), (rel_err(got, want), seed, dtype, cuts, cfg)
        other = random_tokens(cfg["vocab"], 30, seed=seed + 1)
        s1, s2 = cache.open(), cache.open()
        out = st.step([StepEntry(s1, other, want=[29]), StepEntry(s2, tokens[:66], want=[65])])
        assert close(out[1:2], want[65:66], dtype, own32=own32[65:66], gauge=got[65:66]), (seed, dtype)
        assert close(out[0:1], plain_logits(cfg2, w, other)[29:30], dtype,
                     own32=plain_logits(cfg2, w, other, None, torch.float32)[29:30],
                     gauge=rounded_logits(cfg2, w, other)[29:30])
        cache.close(s1); cache.close(s2)


@pytest.mark.parametrize("name,dtype", [("S", "float32"), ("W", "bfloat16")])
def test_trace_replay_through_the_program(tmp_path_factory, tmp_path, name, dtype):
    """bin/trace_run, the program a user runs: a request with its last tokens one by one, and a batch of unequal
    lengths decoded together while the shorter ones end; places where nothing is wanted."""
    from test_gpu_replay import Trace
    folder = make_folder(tmp_path_factory.getbasetemp(), name, dtype)
    cfg, w = read_folder(folder)
    lens = [150, 33, 97, 1]
    reqs = {f"r{i}": random_tokens(cfg["vocab"], n, seed=40 + i) for i, n in enumerate(lens)}
    oracle = {k: plain_logits(cfg, w, t) for k, t in reqs.items()}
    got_rows, want_rows = [], []
    tr = Trace(folder, dtype, tmp_path / "out", max_tokens=192 + 64 + 128 + 64)
    try:
        t = reqs["r0"]                                                   # the tail one by one
        cut = len(t) - 40
        assert tr.step([{"id": "d", "tokens": t[:cut], "want": []}]) is None
        for i in range(cut, len(t)):
            got = tr.step([{"id": "d", "tokens": [t[i]], "want": [0] if i % 3 else []}], end=["d"] if i == len(t) - 1 else [])
            if i % 3:
                got_rows.append(torch.from_numpy(got)); want_rows.append(oracle["r0"][i:i + 1])
        batch = ["r3", "r1", "r2", "r0"]                                 # together; the shorter ones end earlier
        pre = {k: max(1, len(reqs[k]) - 12) for k in batch}
        got = tr.step([{"id": k + "b", "tokens": reqs[k][:pre[k]], "want": [pre[k] - 1]} for k in batch],
                      end=[k + "b" for k in batch if pre[k] == len(reqs[k])])
        for j, k in enumerate(batch):
            got_rows.append(torch.from_numpy(got[j:j + 1])); want_rows.append(oracle[k][pre[k] - 1:pre[k]])
        pos = dict(pre)
        live = [k for k in batch if pre[k] < len(reqs[k])]
        while live:
            ending = [k for k in live if pos[k] + 1 == len(reqs[k])]
            got = tr.step([{"id": k + "b", "tokens": [reqs[k][pos[k]]], "want": [0]} for k in live],
                          end=[k + "b" for k in ending])
            for j, k in enumerate(live):
                got_rows.append(torch.from_numpy(got[j:j + 1])); want_rows.append(oracle[k][pos[k]:pos[k] + 1])
                pos[k] += 1
            live = [k for k in live if k not in ending]
    finally:
        tr.close()
    assert close(torch.cat(got_rows), torch.cat(want_rows), dtype), rel_err(torch.cat(got_rows), torch.cat(want_rows))
