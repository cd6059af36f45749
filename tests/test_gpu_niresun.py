"""The Niresun decoder through the framework against the plain implementation (tests/plain_niresun.py): each mechanism
alone, whole prompts layer by layer, portions, decoding, unequal batches, reuse of slots, pages and states, far keys, chunk
and page borders made to stand out, the first tokens, other sizes, the entry point, the replay program."""
import math
import os

import pytest
import torch

import plain_niresun as plain
from helpers import random_tokens, read_folder, rel_err
from niresun_cases import (CASES, chunked, draw_case, layer, left, make_folder, mamba, model, pair, plain_logits, right, rot,
                           rounded_logits, write_case)
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


def _check_status():
    from gogguf_b200.csrc.tcgen05_gemm import check_status
    check_status(torch.device(DEV))


# ----------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("T,H", [(1, 64), (5, 77), (130, 320), (3, 4100)])
def test_dynamic_tanh(T, H):
    K = _K()
    g = _gen(H)
    x, w, b = torch.randn(T, H, generator=g) * 4, torch.randn(H, generator=g), torch.randn(H, generator=g)
    want = torch.tanh(0.7 * x.double()) * w.double() + b.double()
    for dt in (torch.float32, torch.bfloat16):
        out = torch.empty(T, H, dtype=dt, device=DEV)
        K.dynamic_tanh(x.to(DEV), 0.7, w.to(DEV), b.to(DEV), out)
        assert rel_err(out, want) < (1e-6 if dt == torch.float32 else 5e-3)
    rows = [T - 1, -1, 0]
    out = torch.full((3, H), 9.0, device=DEV)
    K.dynamic_tanh(x.to(DEV), 0.7, w.to(DEV), b.to(DEV), out, _i32(rows))
    assert rel_err(out[0], want[T - 1]) < 1e-6 and float(out[1].abs().max()) == 0.0 and rel_err(out[2], want[0]) < 1e-6


@pytest.mark.parametrize("N,K_", [(384, 264), (1000, 512), (2048, 1024), (72, 80), (132, 64)])
def test_a_product_leaves_the_rows_behind_the_next_norm(N, K_):
    """Every form of the product (decode with and without a K split, prompts with and without one, few columns): it adds
    into the residual and leaves the dynamic tanh of the updated rows."""
    from gogguf_b200.csrc import tcgen05_gemm as TG
    from gogguf_b200.parts.base import Linear, NormedRows, Runtime, Workspace
    g = _gen(N + K_)
    w = (torch.randn(N, K_, generator=g) * 0.1).to(torch.bfloat16)
    rt = Runtime(dtype=torch.bfloat16, device=torch.device(DEV))
    ws = Workspace(rt.device)
    lin = Linear(w, rt)
    nw, nb = torch.randn(N, generator=g).to(DEV), torch.randn(N, generator=g).to(DEV)

    class Norm:
        emit = (0.6, nw, nb)
    for m in (1, 7, 33, 100, 128, 129, 300, 700, 1100):
        x = torch.randn(m, K_, generator=g).to(torch.bfloat16)
        res = torch.randn(m, N, generator=g)
        want = res.double() + x.double() @ w.double().t()
        acc, ahead = res.to(DEV), NormedRows(torch.full((m, N), 7.0, dtype=torch.bfloat16, device=DEV))
        lin(x.to(DEV), acc, accumulate=True, ws=ws, emit=ahead)
        assert not ahead.fresh and float((ahead.rows - 7.0).abs().max()) == 0.0       # nobody's turn: nothing is written
        acc, ahead.norm = res.to(DEV), Norm
        lin(x.to(DEV), acc, accumulate=True, ws=ws, emit=ahead)
        assert ahead.fresh == (m <= 128) and rel_err(acc, want) < 3e-5, m
        if m > 128:                                  # the product can, a norm kernel is faster
            acc = res.to(DEV)
            scratch = torch.empty(max(1, TG.pair_scratch_elems(m, N, K_)), device=DEV)
            TG.gemm_tc_norm(x.to(DEV), w.to(DEV), acc, accumulate=True, out_xhat=ahead.rows, out_norm=Norm.emit, scratch=scratch)
            assert rel_err(acc, want) < 3e-5, m
        assert rel_err(ahead.rows, torch.tanh(0.6 * want) * nw.double().cpu() + nb.double().cpu()) < 5e-3, m
    _check_status()


@pytest.mark.parametrize("I,W", [(40, 64), (128, 96), (512, 256), (704, 384)])
def test_gelu_gated_unit(I, W):
    """The stand-alone kernel and the product with the unit in its epilogue, every form."""
    from gogguf_b200.config.spec import PartSpec
    from gogguf_b200.engine.step import StepContext
    from gogguf_b200.parts.base import Runtime, Workspace
    from gogguf_b200.parts.feedforward import SwiGLU
    g = _gen(I)
    w = {"gate": torch.randn(I, W, generator=g) * 0.15, "up": torch.randn(I, W, generator=g) * 0.15,
         "down": torch.randn(W, I, generator=g) * 0.1}
    spec = PartSpec(kind="swiglu", params=dict(hidden_size=W, intermediate_size=I, activation="gelu_tanh",
                                               names=dict(gate="gate", up="up", down="down")))
    for dt, fast in ((torch.float32, False), (torch.bfloat16, True), (torch.bfloat16, False)):
        rt = Runtime(dtype=dt, device=torch.device(DEV), fast=fast)
        wd = {n: t.to(dt) for n, t in w.items()}
        part = SwiGLU(spec, wd, rt)
        assert (part.fused is not None) == (fast and I % 64 == 0 and I >= 128)
        for T in (1, 9, 70, 129, 400):
            h = (torch.randn(T, W, generator=g) * 2).to(dt)
            want = plain.feed_forward({n: t.double() for n, t in wd.items()}, "", h.double())
            ctx = StepContext(runtime=rt, ws=Workspace(rt.device), n_tokens=T, n_seqs=1, tokens=None, positions=None,
                              seq_of_token=None, cu_seqlens=None, slots=None, ctx_lens=None, page_tables={}, max_new=T, max_ctx=T,
                              decode=False)
            out = torch.zeros(T, W, device=DEV)
            part.forward(h.to(DEV), out, ctx)
            assert rel_err(out, want) < (3e-6 if dt == torch.float32 else 1e-2), (dt, fast, T)


@pytest.mark.parametrize("P,T,H", [(2, 5, 64), (1, 3, 77), (3, 130, 320), (4, 2, 2052), (2, 9, 2048), (2, 3, 4096), (1, 2, 1500),
                                   (2, 2, 4104), (2, 3, 50)])
def test_sum_of_normed_parts(P, T, H):
    K = _K()
    g = _gen(P * H)
    x, y, w = torch.randn(T, H, generator=g), torch.randn(P, T, H, generator=g) * 3, torch.randn(P, H, generator=g)
    y[0, T - 1] = 0.0                                              # a part that says nothing adds nothing
    eps = [1e-5, 1e-2, 1e-6, 0.3][:P]
    nw, nb = torch.randn(H, generator=g), torch.randn(H, generator=g)
    want = x.double() + sum(plain.unit(y[k].double(), eps[k]) * w[k].double() for k in range(P))
    for dt in (None, torch.float32, torch.bfloat16):
        xd, yd = x.to(DEV), y.to(DEV)
        out = None if dt is None else torch.empty(T, H, dtype=dt, device=DEV)
        zero = dt != torch.bfloat16
        K.normed_sum(xd, yd, w.to(DEV), eps, out, None if dt is None else (0.4, nw.to(DEV), nb.to(DEV)), zero_y=zero)
        assert rel_err(xd, want) < 2e-6 and (float(yd.abs().max()) == 0.0 if zero else torch.equal(yd.cpu(), y))
        if dt is not None:
            assert rel_err(out, torch.tanh(0.4 * want) * nw.double() + nb.double()) < (2e-6 if dt == torch.float32 else 5e-3)


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nq,nkv,d,dv,taps,rdims,unit,temp", [
    (6, 2, 12, 20, 4, 0, True, (0.5, 7.0)), (4, 4, 64, 64, 2, 0, True, (0.2, 64.0)), (3, 1, 18, 10, 0, 6, False, None),
    (2, 1, 17, 9, 1, 0, True, (1.0, 1.0)), (8, 2, 128, 96, 9, 64, True, (0.1, 3.0)), (1, 1, 16, 16, 3, 16, False, None)])
def test_preparation_of_q_k_and_v(dt, nq, nkv, d, dv, taps, rdims, unit, temp):
    """Convolution over time, unit heads, temperature, a partial rotation, the cache's rows where the page table says: in
    portions that go on from the convolution's state, in decode steps that move it on themselves; a padding row touches
    nothing; the columns of a wider row."""
    K = _K()
    g = _gen(nq * d + dv)
    cols, eps = (nq + nkv) * d + nkv * dv, 1e-4
    long = nq in (4, 8)                            # steps of many rows take the form with several tokens a thread
    lens = (700, 7) if long else (150, 7)
    rows = [torch.randn(n, cols, generator=g).to(dt) for n in lens]
    cw = torch.randn(cols, taps, generator=g) if taps else None
    coef, every = temp or (0.0, 1.0)
    ro = dict(dims=rdims, base=900.0) if rdims else None
    want = []
    for r in rows:
        n = r.shape[0]
        u = plain.causal_conv(r.double(), cw.double()) if taps else r.double()
        q, k, v = u.split([nq * d, nkv * d, nkv * dv], dim=1)
        q, k = q.reshape(n, nq, d), k.reshape(n, nkv, d)
        if unit:
            q, k = plain.unit(q, eps), plain.unit(k, eps)
        if temp:
            q = q * plain.query_temperature(n, coef, every)[:, None, None]
        if ro:
            q, k = plain.rotate_halves(q, ro), plain.rotate_halves(k, ro)
        want.append((q.reshape(n, -1), k, v.reshape(n, nkv, dv)))
    slots = [2, 0]
    state = torch.zeros(3, max(taps - 1, 1), cols, device=DEV) if taps > 1 else None
    order = torch.randperm(24, generator=g).tolist()
    table = [order[:11], order[11:22]]
    kp = torch.full((24, nkv, PS, d), 7.0, dtype=dt, device=DEV)
    vp = torch.full((24, nkv, PS, dv), 7.0, dtype=dt, device=DEV)
    tol = 3e-6 if dt == torch.float32 else 6e-3
    at = [0, 0]
    for new in ((lens[0] - 80, 1), (2, 3), (1, 1), (1, 1), (76, 1)):
        cu, sot = _batch(new)
        T = sum(new)
        pos = [at[b] + i for b, n in enumerate(new) for i in range(n)]
        x = torch.cat([rows[b][at[b]:at[b] + n] for b, n in enumerate(new)])
        wide = torch.full((T, cols + 24), 3.0, dtype=dt)
        wide[:, 8:8 + cols] = x
        wide = wide.to(DEV)
        q_out = torch.empty(T, nq * d, dtype=dt, device=DEV)
        cos = sin = None
        if ro:
            ang = torch.tensor(pos, dtype=torch.float64)[:, None] * plain.frequencies(ro)[None]
            cos, sin = torch.cos(ang).float().to(DEV), torch.sin(ang).float().to(DEV)
        K.qkv_prep(wide[:, 8:8 + cols], q_out, None, None, eps, 1 if unit else 0, cos, sin, _i32(pos), sot, _i32(table), PS, kp, vp, T, nq,
                   nkv, d, dv, rdims, conv=cw.t().contiguous().to(DEV) if taps else None, conv_state=state, cu_seqlens=cu,
                   slots=_i32(slots), n_seqs=2, max_new=max(new), coef=coef, every=every)
        ref = torch.cat([want[b][0][at[b]:at[b] + n] for b, n in enumerate(new)])
        assert rel_err(q_out, ref) < tol, (new, rel_err(q_out, ref))
        at = [a + n for a, n in zip(at, new)]
    seen = torch.zeros(24, PS, dtype=torch.bool)
    for b, n in enumerate(lens):
        for p in range(n):
            pg, sl = table[b][p // PS], p % PS
            seen[pg, sl] = True
        got_k = torch.cat([kp[pg].permute(1, 0, 2) for pg in table[b]])[:n]
        got_v = torch.cat([vp[pg].permute(1, 0, 2) for pg in table[b]])[:n]
        assert rel_err(got_k, want[b][1]) < tol and rel_err(got_v, want[b][2]) < tol
        if taps > 1:
            assert rel_err(state[slots[b]], rows[b][-(taps - 1):].double() if n >= taps - 1 else torch.cat(
                [torch.zeros(taps - 1 - n, cols, dtype=torch.float64), rows[b].double()])) < 1e-6
    assert float((kp.float().cpu().permute(0, 2, 1, 3)[~seen] - 7.0).abs().max()) == 0.0
    assert float((vp.float().cpu().permute(0, 2, 1, 3)[~seen] - 7.0).abs().max()) == 0.0
    if taps > 1:
        assert float(state[1].abs().max()) == 0.0
        before = [t.clone() for t in (kp, vp, state)]
        cu, sot = _batch((1, 1))
        sot[:] = -1
        K.qkv_prep(wide[:2, 8:8 + cols], q_out[:2], None, None, eps, 1 if unit else 0, cos, sin, _i32([0, 0]), sot, _i32(table), PS, kp, vp,
                   2, nq, nkv, d, dv, rdims, conv=cw.t().contiguous().to(DEV), conv_state=state, cu_seqlens=cu, slots=_i32([0, 0]),
                   n_seqs=2, max_new=1, coef=coef, every=every)
        assert all(torch.equal(a, b) for a, b in zip(before, (kp, vp, state))) and float(q_out[:2].abs().max()) == 0.0


@pytest.mark.parametrize("dt,odt", [(torch.float32, torch.float32), (torch.bfloat16, torch.float32), (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("C,taps", [(64, 4), (36, 2), (260, 3), (33, 4), (40, 6), (24, 1)])
def test_convolution_of_columns(dt, odt, C, taps):
    """Short and long steps (a row, or eight, a thread; one channel or four), sequences that start inside a group of rows,
    single tokens that move the state on themselves, silu or not, both output types."""
    K = _K()
    g = _gen(C + taps)
    lens, slots = (1090, 3, 40), [1, 3, 0]
    rows = [torch.randn(n, C, generator=g).to(dt) for n in lens]
    w, b = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    for act in (0, 1):
        want = [plain.causal_conv(r.double(), w.double(), b) for r in rows]
        want = [plain.silu(v) for v in want] if act else want
        state = torch.zeros(4, taps - 1, C, device=DEV) if taps > 1 else None
        at = [0, 0, 0]
        for new in ((1061, 1, 6), (1, 1, 1), (27, 0, 32), (1, 1, 1)):
            own = [i for i in range(3) if new[i]]
            cu, sot = _batch([new[i] for i in own])
            T = sum(new)
            wide = torch.full((T, C + 16), 3.0, dtype=dt)
            wide[:, 8:8 + C] = torch.cat([rows[i][at[i]:at[i] + new[i]] for i in own])
            out = torch.full((T, C), 9.0, dtype=odt, device=DEV)
            K.column_conv(wide.to(DEV)[:, 8:8 + C], out, w.t().contiguous().to(DEV), b.to(DEV), None, state, cu, _i32([slots[i] for i in own]),
                          sot, T, len(own), act=act, max_new=max(new))
            ref = torch.cat([want[i][at[i]:at[i] + new[i]] for i in own])
            assert rel_err(out, ref) < (2e-6 if odt == torch.float32 else 6e-3), (new, act)
            at = [a + n for a, n in zip(at, new)]
        for i in range(3):
            if taps > 1:
                assert torch.equal(state[slots[i]].cpu(), rows[i].float()[-(taps - 1):] if lens[i] >= taps - 1 else torch.cat(
                    [torch.zeros(taps - 1 - lens[i], C), rows[i].float()]))


def _attention_reference(q, k, v, gate, pos, lens, scale, chunk, window, out_scale=1.0):
    """q [T, H, d] of the step's tokens, k[b] [n, G, d] and v[b] [n, G, dv] everything each sequence has cached."""
    out, t = [], 0
    H = q.shape[1]
    for b, n in enumerate(lens):
        own = [h // (H // k[b].shape[1]) for h in range(H)]
        for _ in range(n):
            p = int(pos[t])
            lo = max(p // chunk * chunk if chunk else 0, p - window + 1 if window else 0)
            s = torch.einsum("hd,jhd->hj", q[t], k[b][lo:p + 1][:, own]) * scale
            out.append(torch.einsum("hj,jhe->he", torch.softmax(s, dim=-1), v[b][lo:p + 1][:, own]).reshape(-1) * out_scale)
            t += 1
    o = torch.stack(out)
    return o if gate is None else o * plain.sigmoid(gate)


@pytest.mark.parametrize("H,G,d,dv,chunk,window,gated", [
    (6, 2, 72, 48, 100, 0, True), (4, 1, 128, 128, 70, 0, True), (8, 2, 64, 64, 0, 0, False), (7, 1, 64, 88, 90, 0, True),
    (4, 4, 40, 128, 64, 0, False), (3, 3, 8, 8, 1, 0, True), (16, 1, 96, 104, 33, 50, True), (2, 1, 120, 24, 1000, 0, True),
    (6, 2, 12, 20, 37, 0, True), (5, 1, 14, 26, 50, 0, False), (20, 1, 64, 64, 90, 0, True)])
def test_attention_of_other_sizes_in_chunks_behind_a_gate(H, G, d, dv, chunk, window, gated):
    """The plain kernel in both dtypes and the tensor-core kernels (prompts, short portions, decode steps with and without
    shares of the pages): key and value sizes of their own, chunks that start inside pages and inside query tiles, chunks
    of one position, windows as well, pages in no particular order, pages before a chunk that are somebody else's."""
    from gogguf_b200.csrc import fast_attention as fa
    K = _K()
    g = _gen(H * d + dv)
    n_pages = 24
    scale = 1.4 / math.sqrt(d)
    perm = torch.randperm(n_pages, generator=g).tolist()
    tab = [perm[0:8], perm[8:16], perm[16:24]]
    kf = torch.randn(n_pages, G, PS, d, generator=g).to(torch.bfloat16)
    vf = torch.randn(n_pages, G, PS, dv, generator=g).to(torch.bfloat16)
    seq = lambda pool, b: torch.cat([pool[p].permute(1, 0, 2) for p in tab[b]]).double()
    ks, vs = [seq(kf, b) for b in range(3)], [seq(vf, b) for b in range(3)]
    done = [0, 0, 0]
    takes = fa.takes(H, G, d, dv)
    assert takes == (d % 8 == 0 and dv % 8 == 0 and H // G <= 16)
    for lens in ((130, 1, 67), (65, 180, 2), (1, 1, 1), (2, 1, 31), (1, 1, 1), (5, 128, 90), (1, 1, 1)):
        cu, sot = _batch(lens)
        T = sum(lens)
        pos = [done[b] + i for b, n in enumerate(lens) for i in range(n)]
        ends = [x + n for x, n in zip(done, lens)]
        # what lies before every query's chunk may have been given away: another sequence's page stands there
        tt = [list(r) for r in tab]
        for b in range(3):
            lo = max(done[b] // chunk * chunk if chunk else 0, done[b] - window + 1 if window else 0)
            for i in range(max(lo, 0) // PS):
                tt[b][i] = 0
        table = _i32(tt)
        q = torch.randn(T, H, d, generator=g).to(torch.bfloat16)
        wide = torch.randn(T, 16 + H * dv + (-H * dv) % 8, generator=g).to(torch.bfloat16)
        want = _attention_reference(q.double(), ks, vs, wide[:, 16:16 + H * dv].double() if gated else None, pos, lens, scale, chunk,
                                    window)
        for dt in (torch.float32, torch.bfloat16):
            o = torch.empty(T, H * dv, dtype=dt, device=DEV)
            K.attention_plain(q.to(dt).to(DEV), kf.to(dt).to(DEV), vf.to(dt).to(DEV), o, _i32(pos), sot, table, PS, T, H, G, d, scale,
                              window, dv=dv, chunk=chunk, gate=wide.to(dt).to(DEV)[:, 16:16 + H * dv] if gated else None)
            assert rel_err(o, want) < (2e-5 if dt == torch.float32 else 6e-3), (lens, dt)
        if takes:
            gate = wide.to(DEV)[:, 16:16 + H * dv] if gated else None
            kw = dict(dv=dv, chunk=chunk, gate=gate)
            args = (q.to(DEV), kf.to(DEV), vf.to(DEV))
            o = torch.full((T, H * dv), 9.0, dtype=torch.bfloat16, device=DEV)
            fa.attn_prefill(*args, o, cu, _i32(ends), sot, table, PS, 3, T // 64 + 3, H, G, d, scale, window, **kw)
            assert rel_err(o, want) < 1.2e-2, (lens, "short portions", rel_err(o, want))
            o = torch.full((T, H * dv), 9.0, dtype=torch.bfloat16, device=DEV)
            fa.attn_prefill_tc(*args, o, cu, _i32(ends), sot, table, PS, T, 3, T // 128 + 3, H, G, d, scale, window, **kw)
            _check_status()
            assert rel_err(o, want) < 1.2e-2, (lens, "prompts", rel_err(o, want))
            if max(lens) == 1:
                for splits in (1, 2, 4):
                    o = torch.full((T, H * dv), 9.0, dtype=torch.bfloat16, device=DEV)
                    fa.attn_decode_tma(*args, o, _i32(pos), sot, table, PS, T, H, G, d, scale, window, splits, cluster=True, **kw)
                    _check_status()
                    assert rel_err(o, want) < 1.2e-2, (lens, "decode", splits, rel_err(o, want))
        done = ends


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,N", [(32, 1), (52, 5), (70, 11), (128, 16), (40, 24), (33, 32), (64, 50), (20, 100), (48, 200)])
def test_selective_scan(dt, C, N):
    """Prompts of unequal lengths walked whole and in chunks, portions and single tokens that go on from the state, slow and
    fast decays, steps near zero and large ones; a padding row leaves zeros and the state alone."""
    K = _K()
    g = _gen(C * N)
    lens, slots = (190, 33), [3, 1]
    D = [dict(x=torch.randn(n, C, generator=g), z=torch.randn(n, C, generator=g), dt=torch.randn(n, C, generator=g) * 2 - 1,
              B=torch.randn(n, N, generator=g), C=torch.randn(n, N, generator=g)) for n in lens]
    for r in D:
        for key in ("x", "z", "B", "C"):
            r[key] = r[key].to(dt)
    A = -torch.exp(torch.randn(C, N, generator=g) * 1.5)
    skip = torch.randn(C, generator=g)
    want = [plain.selective_scan(r["x"].double(), plain.softplus(r["dt"].double()), A.double(), r["B"].double(), r["C"].double(),
                                 skip.double()) * plain.silu(r["z"].double()) for r in D]
    tol = 3e-6 if dt == torch.float32 else 6e-3
    off = 6
    for plan in (((190, 33),), ((130, 1), (1, 1), (1, 1), (2, 17), (56, 13))):
        for chunk in ((0, 64) if len(plan) == 1 else (0,)):
            state = torch.zeros(4, C, N, device=DEV)
            at = [0, 0]
            for new in plan:
                cu, sot = _batch(new)
                T = sum(new)
                part = lambda key: torch.cat([r[key][a:a + n] for r, a, n in zip(D, at, new)])
                xz = torch.cat([part("x"), part("z")], dim=1).to(DEV)
                bc = torch.cat([torch.ones(T, off, dtype=dt), part("B"), part("C")], dim=1).to(DEV)
                out = torch.full((T, C), 9.0, dtype=dt, device=DEV)
                scratch = torch.full((K.selective_scan_scratch(T, 2, C, N, chunk),), 1e30, device=DEV) if chunk else None
                K.selective_scan(xz[:, :C], xz[:, C:], bc, off, off + N, part("dt").to(DEV), out, state, cu, _i32(slots), sot, A.to(DEV),
                                 skip.to(DEV), T, 2, chunk=chunk, scratch=scratch, max_new=max(new))
                ref = torch.cat([w[a:a + n] for w, a, n in zip(want, at, new)])
                assert rel_err(out, ref) < tol, (new, chunk, rel_err(out, ref))
                at = [a + n for a, n in zip(at, new)]
            assert float(state[[0, 2]].abs().max()) == 0.0
    cu, sot = _batch((1, 1))
    sot[1] = -1
    before = state.clone()
    out = torch.full((2, C), 9.0, dtype=dt, device=DEV)
    K.selective_scan(xz[:2, :C], xz[:2, C:], bc[:2], off, off + N, D[0]["dt"][:2].to(DEV), out, state, cu, _i32([3, 0]), sot,
                     A.to(DEV), skip.to(DEV), 2, 2)
    assert float(out[1].abs().max()) == 0.0 and torch.equal(state[[0, 1, 2]], before[[0, 1, 2]]) and not torch.equal(state[3], before[3])
    after, out1 = state.clone(), out.clone()                       # the form for a token each
    state.copy_(before)
    out.fill_(9.0)
    K.selective_scan(xz[:2, :C], xz[:2, C:], bc[:2], off, off + N, D[0]["dt"][:2].to(DEV), out, state, cu, _i32([3, 0]), sot,
                     A.to(DEV), skip.to(DEV), 2, 2, max_new=1)
    assert rel_err(out, out1.double()) < tol and rel_err(state, after.double()) < 1e-5 and torch.equal(state[[0, 1, 2]], before[[0, 1, 2]])
    assert float(out[1].abs().max()) == 0.0


@pytest.mark.parametrize("H,d,dv,cap,shift", [(3, 10, 14, 6.0, 0.0), (1, 16, 16, 1.0, 0.0), (4, 64, 128, 12.0, 0.0), (2, 128, 128, 15.0, 3.0),
                                              (6, 24, 40, 20.0, -6.0), (2, 72, 64, 30.0, 8.0), (5, 18, 22, 15.0, 2.0), (2, 8, 8, 5.0, 0.0),
                                              (1, 150, 200, 8.0, 0.0), (1, 300, 300, 8.0, 0.0)])
def test_matrix_memory(H, d, dv, cap, shift):
    """Both forms against the recurrence written out: prompts of unequal lengths, portions and single tokens that go on from
    the states, gates that forget at once and that never do, inputs far below and far above what is there (`shift`)."""
    K = _K()
    g = _gen(H * d + dv)
    lens, slots, eps = (200, 70), [2, 0], 1e-5
    width = 2 * H * (d + dv)
    off = (0, H * d, 2 * H * d, H * (2 * d + dv))
    for dt in (torch.float32, torch.bfloat16):
        rows = [torch.randn(n, width + 8, generator=g).to(dt) for n in lens]
        zi = [torch.randn(n, H, generator=g) * 3 + shift for n in lens]
        zf = [torch.randn(n, H, generator=g) * 4 + 2 for n in lens]
        w = torch.randn(H * dv, generator=g)
        want = []
        for r, a, f in zip(rows, zi, zf):
            n, x = r.shape[0], r.double()
            q, k, v, gt = (x[:, o:o + H * e] for o, e in zip(off, (d, d, dv, dv)))
            i = cap * torch.tanh(a.double() / cap)
            lf = -plain.softplus(-cap * torch.tanh(f.double() / cap))
            o = plain.memory_scan(q.reshape(n, H, d) * d ** -0.5, k.reshape(n, H, d), v.reshape(n, H, dv), i, lf)
            want.append(plain.unit(o, eps).reshape(n, -1) * w.double() * plain.sigmoid(gt))
        chunks = dt == torch.bfloat16 and K.memory_chunks_takes(d, dv)
        for plan in (((200, 70),), ((130, 1), (1, 1), (1, 1), (2, 66), (66, 1)), ((64, 64), (128, 2), (8, 4))):
            for form in ("scan", "chunks") if chunks else ("scan",):
                states = tuple(torch.zeros(3, *s, device=DEV) for s in ((H, d, dv), (H, d), (H,)))
                at = [0, 0]
                for new in plan:
                    cu, sot = _batch(new)
                    T = sum(new)
                    cat = lambda v: torch.cat([r[a:a + n] for r, a, n in zip(v, at, new)]).to(DEV)
                    gates = torch.cat([cat(zi), cat(zf), torch.ones(T, 3, device=DEV)], dim=1)
                    x, out = cat(rows), torch.full((T, H * dv), 9.0, dtype=dt, device=DEV)
                    args = (states, cu, _i32(slots), sot, w.to(DEV), T, 2, H, d, dv, d ** -0.5, cap, eps)
                    if form == "chunks" and max(new) > 1:
                        scratch = torch.full((K.memory_chunks_scratch(T, 2, H, d, dv),), 1e30, device=DEV)
                        K.memory_chunks(x, off, gates[:, :H], gates[:, H:2 * H], out, scratch, *args)
                    else:
                        K.memory_scan(x, off, gates[:, :H], gates[:, H:2 * H], out, *args)
                    ref = torch.cat([r[a:a + n] for r, a, n in zip(want, at, new)])
                    tol = 1e-4 if dt == torch.float32 else 8e-3
                    assert rel_err(out, ref) < tol, (dt, form, new, rel_err(out, ref))
                    at = [a + n for a, n in zip(at, new)]
                assert all(float(s[1].abs().max()) == 0.0 for s in states)
        cu, sot = _batch((1, 1))
        sot[0] = -1
        before = [s.clone() for s in states]
        out = torch.full((2, H * dv), 9.0, dtype=dt, device=DEV)
        K.memory_scan(x[:2], off, gates[:2, :H], gates[:2, H:2 * H], out, states, cu, _i32([0, 2]), sot, w.to(DEV), 2, 2, H, d, dv,
                      d ** -0.5, cap, eps)
        assert float(out[0].abs().max()) == 0.0 and all(torch.equal(a[:2], b[:2]) for a, b in zip(before, states))
        assert not torch.equal(before[0][2], states[0][2])


def test_both_forms_of_the_memory_leave_the_same_states():
    K = _K()
    g = _gen(3)
    H, d, dv, n = 3, 40, 72, 150
    off = (0, H * d, 2 * H * d, H * (2 * d + dv))
    x = torch.randn(n, 2 * H * (d + dv), generator=g).to(torch.bfloat16).to(DEV)
    gates = (torch.randn(n, 2 * H, generator=g) * 2).to(DEV)
    cu, sot = _batch((n,))
    res = []
    for form in ("scan", "chunks"):
        states = tuple(torch.zeros(1, *s, device=DEV) for s in ((H, d, dv), (H, d), (H,)))
        out = torch.empty(n, H * dv, dtype=torch.bfloat16, device=DEV)
        args = (states, cu, _i32([0]), sot, torch.ones(H * dv, device=DEV), n, 1, H, d, dv, d ** -0.5, 9.0, 1e-5)
        if form == "scan":
            K.memory_scan(x, off, gates[:, :H], gates[:, H:], out, *args)
        else:
            K.memory_chunks(x, off, gates[:, :H], gates[:, H:], out, torch.empty(K.memory_chunks_scratch(n, 1, H, d, dv), device=DEV), *args)
        res.append(states)
    for a, b in zip(*res):
        assert rel_err(b, a.double()) < 3e-5, rel_err(b, a.double())


# ----------------------------------------------------------------------------------------------- layers and models
def _one_layer(mixer, ff=None, width=64, vocab=61, eps=1e-5):
    return model(vocab, width, eps, [layer(mixer, ff)])


ALONE = {
    "scan": _one_layer(mamba(52, 5, 3, 4)),
    "scan_wide": _one_layer(mamba(256, 16, 16, 4), width=128),
    "scan_one_tap": _one_layer(mamba(40, 20, 1, 1)),
    "chunked": _one_layer(chunked(6, 2, 12, 20, 0.3, 37, rot(6, 10000.0, (4.0, 1.0, 4.0, 64)))),
    "chunked_wide": _one_layer(chunked(8, 2, 64, 128, 0.125, 90, rot(32, 500.0, (8.0, 1.0, 2.0, 32))), width=128),
    "chunked_unstretched": _one_layer(chunked(4, 1, 128, 128, 0.1, 64, rot(128, 1e5)), width=128),
    "chunked_unrotated": _one_layer(chunked(2, 2, 16, 8, 0.3, 50, None)),
    "chunked_long_heads": _one_layer(chunked(3, 1, 136, 200, 0.1, 70, rot(100, 1e4))),
    "parallel": _one_layer(pair(left(6, 2, 12, 20, 0.3, 4, (0.5, 7.0)), right(3, 10, 14, 6.0))),
    "parallel_wide": _one_layer(pair(left(8, 2, 64, 64, 0.2, 4, (0.3, 20.0)), right(4, 64, 128, 12.0)), width=128),
    "parallel_one_tap": _one_layer(pair(left(2, 1, 32, 48, 1.0, 1, (1.0, 1.0)), right(2, 32, 24, 2.0))),
    "dense": _one_layer(mamba(8, 1, 1, 1), 100),
    "dense_wide": _one_layer(mamba(8, 1, 1, 1), 320, width=128),
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


def test_which_kernels_the_wide_model_takes(tmp_path_factory, monkeypatch):
    """Every product on the tensor cores, attention and the memory in their tensor-core forms, and no norm kernel between
    the step's first and its last: the products before them leave the finished rows."""
    from gogguf_b200.engine import StepEntry
    folder = make_folder(tmp_path_factory.getbasetemp(), "W", "bfloat16")
    m, cache, st = load(folder, "bfloat16")
    K = _K()
    for b in m.blocks:
        assert b.normed_ahead
        for x in [p for p, _, _ in b.mixer.members] if hasattr(b.mixer, "members") else [b.mixer]:
            assert x.o.tensor_core
            if hasattr(x, "qkv"):
                assert x._fast is not None and x.qkv.tensor_core
            elif hasattr(x, "norm_weight"):
                assert x._chunked and K.memory_chunks_takes(x.d, x.dv) and x.proj_gates.tensor_core
            else:
                assert x.dt.tensor_core and x.x_proj.tensor_core
    calls = {}
    for n in ("dynamic_tanh", "normed_sum", "attention_plain", "memory_chunks", "memory_scan", "selective_scan"):
        real = getattr(K, n)
        monkeypatch.setattr(K, n, lambda *a, _r=real, _n=n, **k: (calls.__setitem__(_n, calls.get(_n, 0) + 1), _r(*a, **k))[1])
    s = cache.open()
    st.step([StepEntry(s, random_tokens(503, 100, 1), want=[99])])
    assert calls == dict(dynamic_tanh=2, normed_sum=2, memory_chunks=2, selective_scan=2), calls
    calls.clear()
    st.step([StepEntry(s, [5], want=[0])])
    assert calls == dict(dynamic_tanh=2, normed_sum=2, memory_scan=2, selective_scan=2), calls
    cache.close(s)


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
    got = run_cut(st_g, cache_g, tokens[:120], [])
    assert close(got, want[:120], dtype, own32=own32[:120], gauge=whole[:120]), rel_err(got, want[:120])
    assert st_g.replays >= 119


@pytest.mark.parametrize("name,dtype", [("S", "float32"), ("S", "bfloat16"), ("W", "bfloat16"), ("ONE", "float32")])
def test_unequal_batches_and_reused_slots_and_pages(tmp_path_factory, name, dtype):
    """Requests of different lengths in one batch, decoded together while the short ones leave; the slots, pages and states
    they give back are taken by the next batch (the cache is sized so that it must)."""
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
def test_long_decoding_across_pages_and_chunks(tmp_path_factory, dtype):
    """A short prompt and 300 decoded tokens: the sequence crosses page and chunk borders, pages go back as chunks end."""
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
CHUNK = 110


def _standout_model(tmp, kind, store):
    """A one-layer model without feed-forward whose weights make one token stand out.  The marked token's input has a
    large component along a direction that every other token's input is orthogonal to, the asking token's along another.
    Attention: one key element of every head copies the marked direction, the same element of every query the asking
    direction, and the scale is large.  Matrix memory: the marked token alone opens the input gate and nothing forgets.
    Selective scan: the marked token alone has a step size and nothing decays, so its numbers stay in the state until the
    asking token reads them."""
    from gogguf_b200.weights.loader import write_model_folder
    W, V = 64, 64
    g = _gen(31)
    embed = torch.randn(V, W, generator=g)
    # the norm is nearly linear here (small alpha), so directions of the embedding are directions of the input
    a = embed[MARKED] / embed[MARKED].norm()
    for j in range(V):
        if j != MARKED:
            embed[j] -= (embed[j] @ a) * a
    mdir = embed[ASKING] / embed[ASKING].norm()
    small = lambda *s: torch.randn(*s, generator=g) * 0.02
    mid = lambda *s: torch.randn(*s, generator=g) * 0.3
    p, alpha = "l0.mix.", 0.01
    w = {"embed": embed, "head": mid(V, W), "final.norm": torch.ones(W), "final.norm.alpha": torch.tensor(0.5), "final.norm.b": small(W),
         "l0.norm1": torch.ones(W) / alpha, "l0.norm1.alpha": torch.tensor(alpha), "l0.norm1.b": torch.zeros(W)}

    def heads(H, G, d, dv):
        q, k = small(H * d, W), small(G * d, W)
        for h in range(H):
            q[h * d + 9] = mdir
        for gg in range(G):
            k[gg * d + 9] = a
        return q, k, mid(G * dv, W)

    if kind == "chunked":
        H, G, d, dv = 4, 2, 16, 24
        mx = chunked(H, G, d, dv, 1.0, CHUNK, rot(8, 10000.0, (2.0, 1.0, 4.0, 64)))
        q, k, v = heads(H, G, d, dv)
        w.update({p + "q": q, p + "k": k, p + "v": v, p + "q.b": small(H * d), p + "k.b": small(G * d), p + "v.b": small(G * dv),
                  p + "g": mid(H * dv, W), p + "o": mid(W, H * dv)})
    elif kind in ("left", "memory"):
        H, G, d, dv, R, rd, rv = 4, 2, 16, 24, 3, 8, 16
        mx = pair(left(H, G, d, dv, 1.0, 2, (0.3, 40.0)), right(R, rd, rv, 25.0))
        q, k, v = heads(H, G, d, dv)
        taps = lambda n: torch.stack([torch.zeros(n), torch.ones(n)], dim=1) + small(n, 2)
        quiet, loud = (1.0, 1e-3) if kind == "left" else (1e-3, 1.0)
        m = {"q": mid(R * rd, W), "k": mid(R * rd, W), "v": mid(R * rv, W), "g": mid(R * rv, W), "o": mid(W, R * rv), "norm": torch.ones(R * rv),
             "i": torch.stack([a * 6.0] * R), "i.b": torch.full((R,), -20.0), "f": small(R, W), "f.b": torch.full((R,), 20.0),
             "out": torch.full((W,), loud)}
        w.update({p + "left.q": q, p + "left.k": k, p + "left.v": v, p + "left.o": mid(W, H * dv), p + "left.out": torch.full((W,), quiet),
                  p + "left.q.conv": taps(H * d), p + "left.k.conv": taps(G * d), p + "left.v.conv": taps(G * dv)})
        w.update({p + "right." + n: t for n, t in m.items()})
    else:
        C, N, R = 48, 6, 4
        mx = mamba(C, N, R, 2)
        x = mid(R + 2 * N, C)
        w.update({p + "in": mid(2 * C, W), p + "conv": torch.stack([torch.zeros(C), torch.ones(C)], dim=1), p + "conv.b": torch.zeros(C),
                  p + "x": x, p + "dt": torch.zeros(C, R), p + "dt.b": torch.full((C,), -14.0), p + "A_log": torch.full((C, N), -9.0),
                  p + "D": small(C), p + "o": mid(W, C)})
        # channel 0 carries the marked direction alone; it alone makes steps
        w[p + "in"][0] = a * 0.8
        x[:R] = 0.0
        x[0, 0] = 2.2
        w[p + "dt"][:, 0] = 1.0
    cfg = model(V, W, 1e-6, [layer(mx, None)])
    folder = os.path.join(str(tmp), f"standout_{kind}_{store}")
    write_model_folder(folder, cfg, {n: t.to(torch.bfloat16 if store == "bfloat16" else torch.float32) for n, t in w.items()})
    return folder


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["chunked", "left", "memory", "scan"])
def test_a_token_far_back_at_borders_and_at_the_start(tmp_path, dtype, kind):
    """The marked token stands once in a long sequence: first, second, around page and chunk borders, hundreds of tokens
    back, just before the end.  The asking token at the end must see it (the same sequence without it gives another
    row), or, in a layer with chunks, must see it just inside its chunk and must not just outside."""
    folder = _standout_model(tmp_path, kind, dtype)
    cfg, w = read_folder(folder)
    m, cache, st = load(folder, dtype)
    for n in (331, 321, 330):                                     # 330 is a chunk's border: the last token is its first
        for marked in (0, 1, 62, 63, 64, 65, 127, 128, 219, 220, 221, 319, n - 2):
            tokens = [t if t not in (MARKED, ASKING) else 7 for t in random_tokens(cfg["vocab"], n, seed=marked)]
            tokens[marked], tokens[-1] = MARKED, ASKING
            without = list(tokens)
            without[marked] = 9
            want = plain_logits(cfg, w, tokens)
            own32 = plain_logits(cfg, w, tokens, None, torch.float32) if dtype == "float32" else want
            moved = rel_err(plain_logits(cfg, w, without)[-1], want[-1])
            if kind == "chunked" and marked // CHUNK != (n - 1) // CHUNK:
                assert moved < 1e-12
            else:
                assert moved > 0.02, (kind, n, marked, moved)
            for cuts in ([n], [n - 1], [marked + 1, n - marked - 2], [n - 40]):
                if min(cuts) < 1 or (n != 331 and len(cuts) == 1 and cuts != [n]):
                    continue
                got = run_cut(st, cache, tokens, cuts)
                rows = [marked, n - 1]
                assert close(got[rows], want[rows], dtype, own32=own32[rows]), (rel_err(got[rows], want[rows]), kind, n, marked, cuts)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_edges_of_chunks_in_prompts_and_in_decoding(tmp_path, dtype):
    """Asking tokens everywhere, one marked token at a chunk's last place, its next one's first, and one further: every
    asking token of the same chunk sees it, the ones beyond do not."""
    folder = _standout_model(tmp_path, "chunked", dtype)
    cfg, w = read_folder(folder)
    m, cache, st = load(folder, dtype)
    n = 2 * CHUNK + 40
    for marked in (CHUNK - 1, CHUNK, CHUNK + 1, 2 * CHUNK - 1, 2 * CHUNK):
        tokens = [ASKING] * n
        tokens[marked] = MARKED
        want = plain_logits(cfg, w, tokens)
        base = plain_logits(cfg, w, [ASKING] * n)
        moved = ((want - base).abs().amax(dim=1) / want.abs().max()) > 0.02
        see = [i for i in range(n) if i >= marked and i // CHUNK == marked // CHUNK]
        assert [i for i in range(n) if moved[i]] == see
        for cuts in ([n], [marked], [CHUNK - 2, 4, CHUNK - 5, 4]):
            got = run_cut(st, cache, tokens, cuts)
            assert close(got, want, dtype, few=False), (rel_err(got, want), marked, cuts)


# ----------------------------------------------------------------------------------------------- entry point, others
def test_greedy_generation_through_the_entry_point(tmp_path_factory):
    import gogguf_b200 as gg
    for name, dtype in (("S", "float32"), ("W", "bfloat16")):
        folder = make_folder(tmp_path_factory.getbasetemp(), name, dtype, std=0.2 if dtype == "float32" else None)
        cfg, w = read_folder(folder)
        prompts = [random_tokens(cfg["vocab"], n, 30 + n) for n in (5, 1, 80)]
        engine = gg.load(folder, gg.LoadOptions(dtype=dtype, max_tokens=1024))
        ctx = engine.new_context()
        out = ctx.generate(prompts, gg.GenerateParams(max_tokens=12, stop_token_ids=[], keep_logits=True))
        rows, refs, own = [], [], []
        for p, r in zip(prompts, out):
            assert len(r.tokens) == 12 and r.prompt_tokens == len(p) and len(r.logits) == 12
            whole = plain_logits(cfg, w, list(p) + r.tokens[:-1])
            whole32 = plain_logits(cfg, w, list(p) + r.tokens[:-1], None, torch.float32)
            for k, row in enumerate(r.logits):
                assert int(row.argmax()) == r.tokens[k]            # greedy: the token is the best of its own row
                rows.append(row)
                refs.append(whole[len(p) - 1 + k])
                own.append(whole32[len(p) - 1 + k])
        assert close(torch.stack(rows), torch.stack(refs), dtype, own32=torch.stack(own)), rel_err(torch.stack(rows), torch.stack(refs))
        # a second round in the same context reuses the slots and pages the first gave back; without kept logits the
        # loop runs a step ahead of the host and drops the step a finished sequence ran too far
        again = ctx.generate(prompts, gg.GenerateParams(max_tokens=12, stop_token_ids=[]))
        assert [r.tokens for r in again] == [r.tokens for r in out]
        stop = out[2].tokens[4]
        third = ctx.generate(prompts, gg.GenerateParams(max_tokens=12, stop_token_ids=[stop]))
        assert third[2].tokens == out[2].tokens[:out[2].tokens.index(stop)]
        ctx.cache.check()
        assert ctx.cache.live_slots == 0


@pytest.mark.parametrize("seed", list(range(16)))
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
        rounded = rounded_logits(cfg2, w, tokens) if dtype == "bfloat16" else None
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
