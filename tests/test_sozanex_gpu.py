"""Sozanex on the GPU against the float64 oracle (tests/sozanex_oracle.py): every mechanism's kernel alone, then the model
through the framework's step function, state manager, decode engine and Generator.  Configurations and weights are made
here; float32 runs are held to a tight bound at every position (only summation order differs), bfloat16 runs to 3 times
what bfloat16 rounding alone does to the logits."""
import ctypes
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import sozanex_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 1e-4
F64 = torch.float64
BF16, F32 = 0, 1      # storage types of the library (AO_LM_BF16, AO_LM_F32)
DTYPES = [torch.float32, torch.bfloat16]


def _lm():
    from torchao_fork_b200 import _lib
    return _lib, _lib.lm()


def _st():
    return torch.cuda.current_stream().cuda_stream


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _p(t):
    return None if t is None else t.data_ptr()


def _dt(dtype):
    return BF16 if dtype == torch.bfloat16 else F32


def _errs(got, ref):
    """Per position: root mean square of the difference (mean over the vocabulary taken off), relative to the reference's spread."""
    got, ref = torch.as_tensor(got).double().cpu(), torch.as_tensor(ref).double().cpu()
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    r = ref - ref.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / r.pow(2).mean(-1).sqrt().clamp_min(1e-30)


def _err(got, ref):
    return float(_errs(got, ref).max())


def _tol(cfg, w, toks, dtype):
    """A bfloat16 run may be 3 times as far from the exact logits as bfloat16 rounding alone moves them."""
    return F32_TOL if dtype == torch.float32 else 3.0 * O.rounding_noise(cfg, w, toks, _err)


def _model(cfg, w, dtype=torch.float32, slots=2, seq=256):
    from torchao_fork_b200._models.sozanex import Sozanex, SozanexArgs
    m = Sozanex(SozanexArgs.from_dict(cfg), w, "cuda", dtype).eval()
    m.setup_caches(slots, seq)
    return m


def _tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=_gen(seed)).tolist()


def _rows(segs):
    """[(slot, first position, rows)] -> per-row slot, pos, back, ahead on the device."""
    slot, pos, back, ahead = [], [], [], []
    for s, p0, c in segs:
        slot += [s] * c
        pos += list(range(p0, p0 + c))
        back += list(range(c))
        ahead += list(range(c - 1, -1, -1))
    return _i32(slot), _i32(pos), _i32(back), _i32(ahead)


def _tiles(segs, tile):
    """Tiles of <= tile rows inside the segments -> (first rows, counts)."""
    tf, tc, at = [], [], 0
    for _, _, c in segs:
        for r in range(0, c, tile):
            tf.append(at + r)
            tc.append(min(tile, c - r))
        at += c
    return _i32(tf), _i32(tc)


def _close(got, ref, tol=2e-5):
    got, ref = got.double().cpu(), ref.double().cpu()
    return bool(torch.isfinite(got).all()) and float((got - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max()))


def _cuts(total, sizes):
    """Portions of the given sizes, repeated, until `total` rows are covered -> [(first, rows)]."""
    out, at, i = [], 0, 0
    while at < total:
        c = min(sizes[i % len(sizes)], total - at)
        out.append((at, c))
        at, i = at + c, i + 1
    return out


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,n", [(1, 3), (33, 7), (128, 5), (2500, 4), (2048, 300), (1030, 301), (16384, 3)])
def test_sublayer_result_enters_through_its_norm_and_the_next_norm_follows(dtype, W, n):
    lib, L = _lm()
    dt, g, eps = _dt(dtype), _gen(W), 1e-3
    x, y = torch.randn(n, W, generator=g) * 3 + 4.0, torch.randn(n, W + 4, generator=g) * 2 - 30.0     # means far from zero
    yb, add = torch.randn(W, generator=g), torch.randn(n, W + 8, generator=g)
    pw, nw = ((1 + 0.3 * torch.randn(W, generator=g)).to(dtype) for _ in range(2))
    out_tol = 3e-5 if dt == F32 else 1e-2
    ycut = y[:, :W].double()
    run = lambda xd, *a: lib.lm_check(L.ao_lm_post_layer_norm_residual(_p(xd), *a, _st()), "post_layer_norm")
    yd, ybd, addd, pwd, nwd = y.cuda(), yb.cuda(), add.cuda(), pw.cuda(), nw.cuda()
    new = lambda: torch.full((n, W + 4), 9.0, device="cuda", dtype=dtype)
    for bias in (True, False):                     # the closing of a sublayer, with and without a projection bias
        xd, out = x.cuda(), new()
        run(xd, _p(yd), W + 4, _p(ybd) if bias else None, _p(pwd), None, 0, 0, _p(nwd), dt, eps, n, W, _p(out), W + 4)
        xs = x.double() + O.layer_norm(ycut + (yb.double() if bias else 0), pw.double(), eps)
        assert _close(xd, xs, 3e-5) and _close(out[:, :W].float(), O.layer_norm(xs, nw.double(), eps), out_tol)
        assert float((out[:, W:].float() - 9).abs().max()) == 0.0
    xd, out = x.cuda(), new()                      # ... with the residual itself as the next product's operand
    run(xd, _p(yd), W + 4, None, _p(pwd), None, 0, 0, None, dt, eps, n, W, _p(out), W + 4)
    xs = x.double() + O.layer_norm(ycut, pw.double(), eps)
    assert _close(xd, xs, 3e-5) and _close(out[:, :W].float(), xs, out_tol)
    xd, out = x.cuda(), new()                      # a pass's input: the sum of two products replaces the residual
    run(xd, _p(yd), W + 4, None, None, _p(addd), W + 8, 1, _p(nwd), dt, eps, n, W, _p(out), W + 4)
    xs = ycut + add[:, :W].double()
    assert _close(xd, xs, 1e-6) and _close(out[:, :W].float(), O.layer_norm(xs, nw.double(), eps), out_tol)
    xd, out = x.cuda(), new()                      # a norm alone leaves the residual as it is; no output: the residual alone
    run(xd, None, 0, None, None, None, 0, 0, _p(nwd), dt, eps, n, W, _p(out), W + 4)
    assert torch.equal(xd.cpu(), x) and _close(out[:, :W].float(), O.layer_norm(x.double(), nw.double(), eps), out_tol)
    run(xd, _p(yd), W + 4, None, _p(pwd), None, 0, 0, None, dt, eps, n, W, None, 0)
    assert _close(xd, x.double() + O.layer_norm(ycut, pw.double(), eps), 3e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,buckets,mp,mc", [(5, 7, 3, 5), (64, 1, 2, 2), (1200, 97, 1, 0), (36, 1009, 10**12 + 39, 10**11 + 3)])
def test_bigram_embedding_in_portions_of_several_sequences(dtype, W, buckets, mp, mc):
    lib, L = _lm()
    dt, V, g = _dt(dtype), 53, _gen(W)
    e = {"scale": 1.7, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}
    table, big = torch.randn(V, W, generator=g).to(dtype), torch.randn(buckets + 1, W, generator=g).to(dtype)
    a, b = torch.randint(0, V, (40,), generator=g).tolist(), torch.randint(0, V, (40,), generator=g).tolist()
    w = {"embed": table.double(), "bigram": big.double()}
    want = {"a": O.embedding({"embedding": e}, w, a), "b": O.embedding({"embedding": e}, w, b)}
    td, bd, last = table.cuda(), big.cuda(), torch.full((4,), 50, dtype=torch.int64, device="cuda")     # slots hold other tokens
    at = {"a": 0, "b": 0}
    for step in ([("a", 17), ("b", 1)], [("b", 1), ("a", 1)], [("a", 2), ("b", 9)], [("b", 29), ("a", 20)]):
        segs = [({"a": 2, "b": 0}[k], at[k], c) for k, c in step]
        toks = sum(({"a": a, "b": b}[k][at[k]:at[k] + c] for k, c in step), [])
        ref = torch.cat([want[k][at[k]:at[k] + c] for k, c in step])
        n = len(toks)
        sd, pd, bk, ad = _rows(segs)
        x, out = torch.zeros(n, W, device="cuda"), torch.zeros(n, W, device="cuda", dtype=dtype)
        tok = torch.tensor(toks, device="cuda")
        lib.lm_check(L.ao_lm_embed_bigram(_p(td), _p(bd), dt, _p(tok), n, W, 1.7, buckets, mp, mc, _p(last), _p(sd), _p(pd), _p(bk), _p(ad),
                                          _p(x), _p(out), _st()), "embed_bigram")
        assert _close(x, ref, 1e-6) and _close(out.float(), ref, 1e-6 if dt == F32 else 1e-2)
        for k, c in step:
            at[k] += c
    assert last.tolist() == [b[-1], 50, a[-1], 50]
    x = torch.zeros(3, W, device="cuda")                  # without a bigram table
    tok = torch.tensor([3, V - 1, 0], device="cuda")
    lib.lm_check(L.ao_lm_embed_bigram(_p(td), None, dt, _p(tok), 3, W, 0.5, 0, 0, 0, None, None, None, None, None, _p(x), None, _st()), "embed")
    assert _close(x, table.double()[[3, V - 1, 0]] * 0.5, 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,dims,pairing", [(4, 2, 12, 8, 8, 1), (3, 1, 7, 5, 6, 1), (20, 5, 64, 48, 64, 1), (2, 2, 16, 16, 0, 1), (1, 1, 2, 1, 2, 1), (5, 5, 300, 4, 200, 1), (3, 3, 10, 6, 4, 0)])
@pytest.mark.parametrize("n", [6, 310])
def test_normed_and_rotated_queries_and_keys(dtype, H, G, d, dv, dims, pairing, n):
    lib, L = _lm()
    dt, g, eps, ring = _dt(dtype), _gen(H + d), 1e-2, 7
    qo, ko, vo = 4, 4 + H * d, 4 + (H + G) * d
    ld = vo + G * dv + 3
    proj = torch.randn(n, ld, generator=g)
    pos = ([0, 1, 5, 300, 70001, 17] * 52)[:n]
    qb, kb, vb, qw, kw = (torch.randn(s, generator=g).to(dtype) for s in (H * d, G * d, G * dv, d, d))
    rot = O.rotary(dims, 900.0) if dims else None
    inv = O.frequencies(rot)[0].float().cuda() if dims else None
    dev = [t.cuda() for t in (proj, qb, kb, vb, qw, kw)]
    pd, sd = _i32(pos), _i32([0] * n)
    qn, kn, vn = torch.zeros(n, H, d, device="cuda"), torch.zeros(n, G, d, device="cuda", dtype=dtype), torch.zeros(n, G * dv, device="cuda", dtype=dtype)
    rk, rv = torch.full((2, ring, G * d), 5.0, device="cuda", dtype=dtype), torch.full((2, ring, G * dv), 5.0, device="cuda", dtype=dtype)

    def run(slot, ring_k, ring_v, rows):
        lib.lm_check(L.ao_lm_qkv_norm_rotary_prep(_p(dev[0]), ld, qo, ko, vo, *(_p(t) for t in dev[1:]), eps, _p(pd), _p(inv), dims, pairing, 1.0, rows,
                                                  H, G, d, G * dv, dt, _p(qn), _p(kn), _p(vn), _p(slot), ring, ring_k, ring_v, _st()), "prep")

    run(sd, None, None, n)
    p, layout = torch.tensor(pos), "half" if pairing else "interleaved"
    # fp32 angles: an angle of 70001 radians is known to 4e-3 at best, whatever computes it
    ref = lambda o, bias, wt, heads: O.rotate(O.rms_norm((proj[:, o:o + heads * d].double() + bias.double()).view(n, heads, d), wt.double(), eps), p, rot, layout)
    rq, rkk = ref(qo, qb, qw, H), ref(ko, kb, kw, G)
    near = p < 1000
    assert _close(qn[near.cuda()], rq[near], 1e-4) and _close(qn, rq, 2e-2)
    assert _close(kn[near.cuda()].float(), rkk[near], 1e-4 if dt == F32 else 1e-2)
    assert _close(vn.float(), proj[:, vo:vo + G * dv].double() + vb.double(), 1e-6 if dt == F32 else 1e-2)
    one = _i32([1])
    k0, v0 = kn[0].clone(), vn[0].clone()
    run(one, _p(rk), _p(rv), 1)                            # one row per sequence: it also enters the ring, and only its row
    assert torch.equal(rk[1, 0].view(G, d), k0) and torch.equal(rv[1, 0], v0)
    assert float((rk[0].float() - 5).abs().max()) == 0.0 and float((rv[1, 1:].float() - 5).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Rq,R,dr,dims,n", [(10, 14, 4, 4, 5), (768, 512, 64, 64, 3), (1, 1, 2, 2, 2), (96, 60, 6, 4, 300), (128, 256, 32, 0, 301)])
def test_latent_norms_rotated_key_part_and_cache_rows(dtype, Rq, R, dr, dims, n):
    lib, L = _lm()
    dt, g, eps, S = _dt(dtype), _gen(R), 1e-3, 330
    qo, ko = 8, 8 + Rq
    ld = ko + R + dr + (-(ko + R + dr)) % 4
    proj, pos = torch.randn(n, ld, generator=g), list(range(11, 11 + n))
    qw, cw = torch.randn(Rq, generator=g).to(dtype), torch.randn(R, generator=g).to(dtype)
    rot = O.rotary(dims, 700.0, ramp=(4.0, 64, 8.0, 1.0)) if dims else None
    f, amp = O.frequencies(rot) if dims else (torch.ones(1), 1.0)
    fd, pd, sd, prd, qwd, cwd = f.float().cuda(), _i32(pos), _i32([1] * n), proj.cuda(), qw.cuda(), cw.cuda()
    z = lambda *s: torch.full(s, 3.0, device="cuda", dtype=dtype)
    cq, c, kr, cc, ck = z(n, Rq), z(n, R), z(n, dr), z(2, S, R), z(2, S, dr)
    lib.lm_check(L.ao_lm_latent_low_prep_store(_p(prd), ld, n, qo, Rq, ko, R, dr, _p(qwd), _p(cwd), dt, eps, dims, _p(fd), amp, _p(pd), _p(sd), S,
                                               _p(cq), _p(c), _p(kr), _p(cc), _p(ck), _st()), "low_prep_store")
    tol = 3e-5 if dt == F32 else 1e-2
    assert _close(cq.float(), O.rms_norm(proj[:, qo:qo + Rq].double(), qw.double(), eps), tol)
    assert _close(c.float(), O.rms_norm(proj[:, ko:ko + R].double(), cw.double(), eps), tol)
    assert _close(kr.float(), O.rotate(proj[:, ko + R:ko + R + dr].double().view(n, 1, dr), torch.tensor(pos), rot, "interleaved")[:, 0], 1e-4 if dt == F32 else 1e-2)
    assert torch.equal(cc[1, 11:11 + n], c) and torch.equal(ck[1, 11:11 + n], kr)
    assert float((cc[0].float() - 3).abs().max()) == 0.0 == float((cc[1, :11].float() - 3).abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,H,R,dv", [(1, 3, 14, 12), (16, 2, 64, 80), (4, 5, 512, 33), (2, 1, 1, 1), (3, 16, 96, 64)])
def test_value_up_projection_with_the_gate(dtype, n, H, R, dv):
    lib, L = _lm()
    dt, g = _dt(dtype), _gen(R)
    ol, uv = torch.randn(n, H, R, generator=g).to(dtype), (torch.randn(H, dv, R, generator=g) / math.sqrt(R)).to(dtype)
    gate = torch.randn(n, H * dv + 5, generator=g) * 4
    old, uvd, gd = ol.cuda(), uv.cuda(), gate.cuda()
    out = torch.full((n, H * dv + 3), 9.0, device="cuda", dtype=dtype)
    ref = torch.einsum("thr,hdr->thd", ol.double(), uv.double()).reshape(n, H * dv)
    tol = 2e-5 if dt == F32 else 1e-2
    for gp, want in ((_p(gd), ref * torch.sigmoid(gate[:, :H * dv].double())), (None, ref)):
        lib.lm_check(L.ao_lm_latent_value_up(_p(old), _p(uvd), dt, n, H, R, dv, gp, H * dv + 5, _p(out), H * dv + 3, _st()), "value_up")
        assert _close(out[:, :H * dv].float(), want, tol)
    lib.lm_check(L.ao_lm_sigmoid_gate_rows(_p(gd), H * dv + 5, n, H * dv, _p(out), H * dv + 3, dt, _st()), "gate_rows")
    assert _close(out[:, :H * dv].float(), ref * torch.sigmoid(gate[:, :H * dv].double()), tol)
    assert float((out[:, H * dv:].float() - 9).abs().max()) == 0.0


@pytest.mark.parametrize("n", [1, 2, 3, 8])
@pytest.mark.parametrize("M,K,pad", [(37, 96, 0), (2048, 2048, 8), (5, 8, 16), (1000, 9216, 0), (4608, 264, 8), (3, 20000, 0)])
def test_products_of_few_rows(n, M, K, pad):
    lib, L = _lm()
    g = _gen(M)
    x, w = torch.randn(n, K + pad, generator=g).bfloat16(), (torch.randn(M, K + pad, generator=g) / math.sqrt(K)).bfloat16()
    xd, wd = x.cuda(), w.cuda()
    torch.cuda.synchronize()
    ref = x[:, :K].double() @ w[:, :K].double().T
    out, ya = torch.full((n, M + 3), 9.0, device="cuda"), torch.full((n, M + 3), 9.0, device="cuda", dtype=torch.bfloat16)
    for o, act in ((out, 0), (ya, 1)):
        lib.lm_check(L.ao_lm_gemv_rows(_p(xd), K + pad, _p(wd), K + pad, n, M, K, act, _p(o), M + 3, _st()), "gemv")
        assert _close(o[:, :M].float(), O.squared_relu(ref) if act else ref, 1e-2 if act else 2e-5)
        assert float((o[:, M:].float() - 9).abs().max()) == 0.0


@pytest.mark.parametrize("n,H,dn,dr,dims,R", [(1, 3, 8, 4, 4, 16), (8, 2, 200, 6, 2, 96), (2, 16, 128, 64, 64, 512), (3, 1, 1, 2, 0, 8)])
def test_query_fold_of_few_rows(n, H, dn, dr, dims, R):
    lib, L = _lm()
    g = _gen(R + dn)
    q, uk = torch.randn(n, H, dn + dr, generator=g), (torch.randn(H, dn, R, generator=g) / math.sqrt(dn)).bfloat16()
    pos = [5, 0, 999, 17, 3, 8, 1, 2][:n]
    rot = O.rotary(dims, 300.0, ramp=(4.0, 64, 8.0, 1.0)) if dims else None
    f, amp = O.frequencies(rot) if dims else (torch.ones(1), 1.0)
    qd, ukd, fd, pd = q.cuda(), uk.cuda(), f.float().cuda(), _i32(pos)
    torch.cuda.synchronize()
    qa, qr = torch.zeros(H, n, R, device="cuda"), torch.zeros(n, H, dr, device="cuda")
    lib.lm_check(L.ao_lm_latent_query_fold(_p(qd), _p(ukd), BF16, n, H, dn, dr, R, dims, _p(fd), amp, _p(pd), _p(qa), _p(qr), _st()), "query_fold")
    assert _close(qa, torch.einsum("thd,hdr->htr", q[..., :dn].double(), uk.double()))
    assert _close(qr, O.rotate(q[..., dn:].double(), torch.tensor(pos), rot, "interleaved"), 1e-4)


@pytest.mark.parametrize("V,ld", [(1, 1), (7, 8), (4096, 4096), (32000, 32001), (128256, 128256)])
def test_greedy_choice_takes_the_first_of_equals(V, ld):
    lib, L = _lm()
    z = torch.randn(3, ld, generator=_gen(V))
    hot = [V - 1, V // 2, min(V - 1, 5)]
    for b, i in enumerate(hot):
        z[b, i] = 50.0
    z[1, -1 if ld == V else V:] = 50.0                      # a later equal one (or one past the vocabulary)
    zd, out = z.cuda(), torch.zeros(3, dtype=torch.int64, device="cuda")
    lib.lm_check(L.ao_lm_argmax(_p(zd), ld, 3, V, _p(out), _st()), "argmax")
    assert out.tolist() == hot


@pytest.mark.parametrize("types", [(F32, F32), (F32, BF16), (BF16, BF16)])
@pytest.mark.parametrize("n,cols", [(3, 37), (2, 4096), (300, 64), (1, 20000)])
def test_squared_relu_rows(types, n, cols):
    lib, L = _lm()
    z = (torch.randn(n, cols, generator=_gen(cols)) * 2).to(torch.float32 if types[0] == F32 else torch.bfloat16)
    zd, out = z.cuda(), torch.zeros(n, cols, device="cuda", dtype=torch.float32 if types[1] == F32 else torch.bfloat16)
    scale = torch.rand(n, generator=_gen(1)).cuda()
    for s in (None, scale):
        lib.lm_check(L.ao_lm_unary_rows(_p(zd), types[0], n, cols, 0, 0.0, _p(s), 1, _p(out), types[1], _st()), "unary")
        ref = O.squared_relu(z.double()) * (1.0 if s is None else s.cpu().double()[:, None])
        assert _close(out.float(), ref, 1e-6 if types[1] == F32 else 1e-2)


def _latent_run(qn, qr, c, kr, uk, uv, cuts, scale, dtype, form, sink, gate, n_split=1, S=256, slot=2, slots=3):
    """Latent attention with a sink and an element-wise gate over one sequence cut into portions, over a full cache of S rows;
    qn [T][H][dn], qr [T][H][dr], c [T][R], kr [T][dr], uk [H][dn][R], uv [H][dv][R], sink [H], gate [T][H dv] -> [T][H dv]."""
    lib, L = _lm()
    T, H, dn = qn.shape
    dr, R, dv = qr.shape[-1], c.shape[-1], uv.shape[1]
    dt = _dt(dtype)
    rows = ctypes.c_int()
    lib.lm_check(L.ao_lm_latent_attention_plan(dt, H, R, dr, ctypes.byref(rows)) if form == "folded" else
                 L.ao_lm_latent_attention_expanded_plan(dt, dn, dr, dv, ctypes.byref(rows)), "plan")
    assert rows.value > 0
    rc, rk = (torch.full((slots, S, k), 50.0, device="cuda", dtype=dtype) for k in (R, dr))   # rubbish that must not be seen
    sk, outs = sink.to(dtype).cuda(), []
    for a, n in cuts:
        segs = [(slot, a, n)]
        sd, pd, bd, ad = _rows(segs)
        tf, tc = _tiles(segs, rows.value)
        cd, kd = c[a:a + n].to(dtype).cuda().contiguous(), kr[a:a + n].to(dtype).cuda().contiguous()
        qrd, gd = qr[a:a + n].float().cuda().contiguous(), gate[a:a + n].float().cuda().contiguous()
        out = torch.zeros(n, H * dv, device="cuda", dtype=dtype)
        if form == "folded":
            qa = torch.einsum("thd,hdr->htr", qn[a:a + n], uk).float().cuda().contiguous()
            ws = torch.zeros(max(16, int(L.ao_lm_latent_attention_workspace_bytes(n, H, R, n_split))), dtype=torch.uint8, device="cuda")
            ws.view(torch.float32)[:] = float("nan")         # shares that see no key must not be read
            ol, uvd = torch.zeros(n, H, R, device="cuda", dtype=dtype), uv.to(dtype).cuda().contiguous()
            lib.lm_check(L.ao_lm_window_latent_attention(_p(qa), _p(qrd), _p(rc), _p(rk), _p(cd), _p(kd), dt, S, _p(sd), _p(pd), _p(bd), _p(tf),
                                                         _p(tc), len(tf), n, H, R, dr, scale, S, _p(sk), None, n_split, _p(ws), ws.numel(),
                                                         _p(ol), _st()), "folded")
            lib.lm_check(L.ao_lm_latent_value_up(_p(ol), _p(uvd), dt, n, H, R, dv, _p(gd), H * dv, _p(out), H * dv, _st()), "value_up")
        else:
            src = _i32([-1 - (slot * S + p) for p in range(a)] + list(range(n)))
            ca, ka = torch.zeros(a + n, R, device="cuda", dtype=dtype), torch.zeros(a + n, dr, device="cuda", dtype=dtype)
            lib.lm_check(L.ao_lm_latent_rows_gather(_p(src), a + n, _p(cd), _p(kd), _p(rc), _p(rk), dt, R, dr, _p(ca), _p(ka), _st()), "gather")
            kv = torch.cat([torch.einsum("tr,hdr->thd", ca.double(), u.cuda()).flatten(1) for u in (uk, uv)], 1).to(dtype).contiguous()
            ld = H * (dn + dv)
            qd, k0 = qn[a:a + n].transpose(0, 1).to(dtype).cuda().contiguous(), _i32([0] * len(tf))
            lib.lm_check(L.ao_lm_gated_latent_attention_expanded(_p(qd), _p(qrd), _p(kv), ld, kv.data_ptr() + kv.element_size() * H * dn, ld, _p(ka),
                                                                 dt, _p(pd), _p(tf), _p(tc), _p(k0), len(tf), n, H, dn, dr, dv, scale, S,
                                                                 _p(sk), _p(gd), H * dv, _p(out), H * dv, _st()), "expanded")
        lib.lm_check(L.ao_lm_ring_append(_p(cd), _p(kd), n, R, dr, S, dt, _p(sd), _p(pd), _p(ad), _p(rc), _p(rk), _st()), "append")
        outs.append(out.float())
    return torch.cat(outs)


def _latent_reference(qn, qr, c, kr, uk, uv, scale, sink, gate):
    T, H, _ = qn.shape
    k = torch.cat([torch.einsum("tr,hdr->thd", c, uk), kr[:, None].expand(T, H, kr.shape[-1])], -1)
    o = O.sink_softmax(torch.cat([qn, qr], -1), k, torch.einsum("tr,hdr->thd", c, uv), scale, sink=sink)
    return o.reshape(T, -1) * torch.sigmoid(gate)


@pytest.mark.parametrize("form,dtype", [("folded", torch.float32), ("folded", torch.bfloat16), ("expanded", torch.bfloat16)])
@pytest.mark.parametrize("H,dn,dr,R,dv", [(3, 16, 16, 24, 32), (1, 32, 16, 96, 16), (6, 16, 32, 64, 80), (18, 16, 16, 128, 16), (2, 64, 48, 500, 128)])
def test_latent_attention_with_sink_and_gate(form, dtype, H, dn, dr, R, dv):
    T, scale, g = 150, 0.1, _gen(H + R)
    rnd = lambda *s: torch.randn(*s, generator=g).bfloat16().double()
    args = rnd(T, H, dn), rnd(T, H, dr), rnd(T, R), rnd(T, dr), rnd(H, dn, R) / math.sqrt(R), (rnd(H, dv, R) / math.sqrt(R)).bfloat16().double()
    sink, gate = torch.linspace(-2.0, 3.0, H).bfloat16().double(), rnd(T, H * dv) * 2
    ref = _latent_reference(*args, scale, sink, gate)
    assert _close(ref, ref) and not _close(_latent_reference(*args, scale, sink - 9, gate), ref, 5e-2)     # the sink shows
    tol = 1e-4 if dtype == torch.float32 else 1.5e-2
    for cuts, ns in (([(0, T)], 1), (_cuts(T, [2, 64, 1, 19]), 3), (_cuts(T, [130, 2]), 1), (_cuts(T, [T - 6, 1, 1, 1, 1, 1, 1]), 8)):
        assert _close(_latent_run(*args, cuts, scale, dtype, form, sink, gate, ns), ref, tol), (cuts[:3], ns)


@pytest.mark.parametrize("form,dtype", [("folded", torch.float32), ("folded", torch.bfloat16), ("expanded", torch.bfloat16)])
@pytest.mark.parametrize("how", ["whole", "portions", "decoded"])
@pytest.mark.parametrize("part", ["latent", "rotated", "sink"])
def test_one_dominant_latent_row_far_away_or_a_dominant_sink(form, dtype, how, part):
    """One row answers one query so strongly that the query returns that row's values, however far away it lies; a row in the
    future leaves no trace; a sink that dominates silences the head."""
    T, H, dn, dr, dv, R, query = 201, 2, 16, 16, 16, 64, 133
    g = _gen(7)
    c = torch.randn(T, R, generator=g).bfloat16().double()
    c[:, 0] = 0
    uk, uv = torch.zeros(H, dn, R, dtype=F64), torch.randn(H, dv, R, generator=g).bfloat16().double() / 8
    uk[:, 0, 0], uv[:, :, 0] = 1.0, 0.0
    cuts = {"whole": [(0, T)], "portions": _cuts(T, [37, 2, 5]), "decoded": [(0, 129)] + [(i, 1) for i in range(129, T)]}[how]
    gate, weak = torch.full((T, H * dv), 40.0, dtype=F64), torch.full((H,), -60.0, dtype=F64)
    for key, seen in ((0, True), (1, True), (64, True), (128, True), (132, True), (133, True), (134, False), (200, False)):
        qn, qr, kr, cc = torch.zeros(T, H, dn, dtype=F64), torch.zeros(T, H, dr, dtype=F64), torch.zeros(T, dr, dtype=F64), c.clone()
        sink = weak
        if part == "rotated":
            qr[query, :, 3], kr[key, 3] = 32.0, 32.0
        else:
            qn[query, :, 0], cc[key, 0] = 32.0, 32.0
        if part == "sink":
            sink = torch.tensor([-60.0, 1500.0], dtype=F64)       # head 1: far above the dominant row's 1024
        got = _latent_run(qn, qr, cc, kr, uk, uv, cuts, 1.0, dtype, form, sink, gate, 3 if how == "decoded" and form == "folded" else 1)[query, dv:]
        val = cc @ uv[1].T
        want = torch.zeros(dv, dtype=F64) if part == "sink" else val[key] if seen else val[:query + 1].mean(0)
        assert _close(got, want, 1e-4 if dtype == torch.float32 else 2e-2), key


def _window_run(q, k, v, cuts, size, scale, dtype, form, n_split=1, single_rows_go_straight_in=True):
    """Window attention of one sequence cut into portions; q [T][H][d], k [T][G][d], v [T][G][dv] -> [T][H dv]."""
    lib, L = _lm()
    T, H, d = q.shape
    G, dv, dt, slot = k.shape[1], v.shape[-1], _dt(dtype), 1
    rows = ctypes.c_int()
    lib.lm_check((L.ao_lm_window_attention_plan if form == "few" else L.ao_lm_window_attention_prompt_plan)(dt, 1, H, G, d, dv, ctypes.byref(rows)), "plan")
    assert rows.value > 0
    rk, rv = torch.full((2, size, G * d), 50.0, device="cuda", dtype=dtype), torch.full((2, size, G * dv), 50.0, device="cuda", dtype=dtype)
    outs = []
    for a, n in cuts:
        sd, pd, bd, ad = _rows([(slot, a, n)])
        tf, tc = _tiles([(slot, a, n)], rows.value)
        qd, kd, vd = q[a:a + n].float().cuda().contiguous(), k[a:a + n].to(dtype).cuda().contiguous(), v[a:a + n].to(dtype).cuda().contiguous()
        out = torch.zeros(n, H * dv, device="cuda", dtype=dtype)

        def append():
            lib.lm_check(L.ao_lm_window_append(_p(kd), _p(vd), n, G * d, G * dv, size, 0, dt, _p(sd), _p(pd), _p(ad), _p(rk), _p(rv), _p(rk), _p(rv), _st()), "append")
        if n == 1 and single_rows_go_straight_in:          # what the preparation kernel does for a step of single rows
            append()
        common = (_p(qd), _p(kd), _p(vd), _p(rk), _p(rv), _p(rk), _p(rv), size, 0, dt, _p(sd), _p(pd), _p(bd), _p(tf), _p(tc), len(tf), 1, H, G, d, dv,
                  size, 0, scale, 0.0, 0, 0.0, 1.0)
        if form == "few":
            ws = torch.zeros(max(16, int(L.ao_lm_window_attention_workspace_bytes(len(tf), 1, H, G, dv, n_split))), dtype=torch.uint8, device="cuda")
            lib.lm_check(L.ao_lm_window_attention(*common, n_split, _p(ws), ws.numel(), _p(out), H * dv, _st()), "window_attention")
        else:
            lib.lm_check(L.ao_lm_window_attention_prompt(*common, _p(out), H * dv, _st()), "window_attention_prompt")
        append()
        outs.append(out.float())
    return torch.cat(outs)


@pytest.mark.parametrize("form,dtype", [("few", torch.float32), ("few", torch.bfloat16), ("prompt", torch.bfloat16)])
@pytest.mark.parametrize("H,G,d,dv,size", [(4, 2, 16, 48, 9), (3, 3, 32, 16, 1), (6, 1, 64, 80, 70), (2, 2, 16, 16, 64)])
def test_window_attention_whole_in_portions_and_decoded(form, dtype, H, G, d, dv, size):
    T, g = 170, _gen(size)
    rnd = lambda *s: torch.randn(*s, generator=g).bfloat16().double()
    q, k, v = rnd(T, H, d), rnd(T, G, d), rnd(T, G, dv)
    ref = O.sink_softmax(q, k, v, 0.3, size).reshape(T, -1)
    for cuts, ns in (([(0, T)], 1), (_cuts(T, [64, 1, 2, 17]), 1), (_cuts(T, [100] + [1] * 70), 2)):
        assert _close(_window_run(q, k, v, cuts, size, 0.3, dtype, form, ns if form == "few" else 1), ref, 1e-4 if dtype == torch.float32 else 1.5e-2), cuts[:3]


@pytest.mark.parametrize("form,dtype", [("few", torch.float32), ("few", torch.bfloat16), ("prompt", torch.bfloat16)])
@pytest.mark.parametrize("how", ["whole", "portions", "decoded"])
def test_one_dominant_key_just_inside_and_just_outside_the_window(form, dtype, how):
    T, d, dv, size, query = 151, 16, 16, 40, 99
    v = torch.randn(T, 1, dv, generator=_gen(3)).bfloat16().double()
    cuts = {"whole": [(0, T)], "portions": _cuts(T, [37, 2, 5]), "decoded": [(0, 38)] + [(i, 1) for i in range(38, T)]}[how]
    for key, seen in ((60, True), (59, False), (99, True), (98, True), (100, False), (0, False), (64, True)):
        q, k = torch.zeros(T, 2, d, dtype=F64), torch.zeros(T, 1, d, dtype=F64)
        q[query, 1, 2], k[key, 0, 2] = 16.0, 16.0
        got = _window_run(q, k, v, cuts, size, 1.0, dtype, form)[query, dv:]
        want = v[key, 0] if seen else v[query - size + 1:query + 1, 0].mean(0)
        assert _close(got, want, 1e-4 if dtype == torch.float32 else 2e-2), key


# ------------------------------------------------------------------------------------------------ the model
def _mixed():     # both mixers, both frequency scalings, a span run twice in the middle, one layer without feed-forward
    return O.model_config([O.attention_layer(heads=2, kv_heads=1, dim=6, vdim=10, size=5, rot=6),
                           O.latent_layer(ramp=(4.0, 24, 4.0, 1.0)), O.attention_layer(bands=(4.0, 64, 1.0, 4.0), ff=0),
                           O.latent_layer(heads=2, ff=24)], loop=(1, 3, 2))


def _ones():      # sizes that are 1 or equal, a window of one token, one bucket, one pass
    return O.model_config([O.attention_layer(heads=1, kv_heads=1, dim=16, vdim=16, size=1, rot=16, ff=16),
                           O.latent_layer(heads=1, dim=16, rot_dim=16, vdim=16, q_rank=16, kv_rank=16, ff=16)],
                          width=16, vocab=16, scale=1.0, bigram=(1, 1, 1), loop=(0, 2, 1))


def _odd():       # odd sizes everywhere, a looped last layer
    return O.model_config([O.latent_layer(heads=5, dim=3, rot_dim=6, vdim=9, q_rank=7, kv_rank=11, ramp=(3.0, 40, 9.0, 2.0), ff=9),
                           O.attention_layer(heads=9, kv_heads=3, dim=5, vdim=7, size=3, rot=2, bands=(2.0, 9, 0.7, 1.2), ff=29)],
                          width=27, vocab=31, eps=1e-3, scale=2.5, bigram=(13, 7, 2), loop=(1, 2, 3))


def _plain():     # no pair table, no loop, no window, no rotation
    return O.model_config([O.attention_layer(size=0, rot=0), O.latent_layer(), O.attention_layer(size=300, kv_heads=4)], bigram=None)


def _tensor():    # head shapes that the tensor-core kernels cover, everything looped
    return O.model_config([O.latent_layer(heads=4, dim=32, rot_dim=16, vdim=48, q_rank=24, kv_rank=64, ramp=(2.0, 50, 8.0, 1.0), ff=64),
                           O.attention_layer(heads=4, kv_heads=1, dim=32, vdim=64, size=33, rot=16, scale=0.2, bands=(4.0, 90, 1.0, 5.0), ff=64),
                           O.attention_layer(heads=2, kv_heads=2, dim=16, vdim=80, size=70, rot=16, ff=0)], width=64, vocab=97, bigram=(201, 17, 3),
                          loop=(0, 3, 2))


CONFIGS = {"mixed": _mixed, "ones": _ones, "odd": _odd, "plain": _plain, "tensor": _tensor}


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompt_and_every_layer_run_against_oracle(name, dtype):
    cfg = CONFIGS[name]()
    w = O.random_weights(cfg, 21)
    toks = _tokens(cfg, 45, 1)
    layers = []
    ref = O.forward(cfg, w, toks, layers_out=layers)
    m = _model(cfg, w, dtype)
    logits, sums = m.step_engine.layer_sums(m.states.slot_of("a"), toks)
    assert _err(logits, ref) < _tol(cfg, w, toks, dtype)
    assert sums.shape[0] == len(layers)
    if dtype == torch.float32:
        for r in range(sums.shape[0]):
            assert _close(sums[r], layers[r], 1e-4), r


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_prefill_equals_token_by_token_and_portions(dtype, name):
    cfg = CONFIGS[name]()
    w = O.random_weights(cfg, 22)
    toks = _tokens(cfg, 70, 2)
    ref, tol = O.forward(cfg, w, toks), _tol(cfg, w, toks, dtype)
    m = _model(cfg, w, dtype)
    eng, st = m.step_engine, m.states
    whole = eng.step([(st.slot_of("w"), toks)], "all")
    assert _err(whole, ref) < tol
    assert _err(torch.cat([eng.step([(st.slot_of("o"), [t])], "all") for t in toks]), ref) < tol
    st.release("w")
    for sizes in ([2], [7, 1, 2, 23], [33, 2], [17]):
        got = torch.cat([eng.step([(st.slot_of("p"), toks[a:a + c])], "all") for a, c in _cuts(len(toks), sizes)])
        assert _err(got, ref) < tol, sizes
        if dtype == torch.float32:
            assert _err(got, whole) < 5e-5, sizes      # the same sums, in another order at most
        st.release("p")


@pytest.mark.parametrize("min_rows", [1, 1000])
def test_either_attention_form_for_every_portion_and_batch(monkeypatch, min_rows):
    """bf16 with head sizes that both kinds of attention kernels cover: every step attends with the tensor-core / expanded forms
    (min_rows 1, also single decoded tokens) or with the others (min_rows 1000, also long portions)."""
    import torchao_fork_b200._models.segment_step as S
    monkeypatch.setattr(S, "PROMPT_MIN_ROWS", min_rows)
    cfg = _tensor()
    w = O.random_weights(cfg, 29)
    a, b = _tokens(cfg, 140, 3), _tokens(cfg, 30, 4)
    ra, rb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    tol = max(_tol(cfg, w, a, torch.bfloat16), _tol(cfg, w, b, torch.bfloat16))
    m = _model(cfg, w, torch.bfloat16, slots=2)
    eng, st = m.step_engine, m.states
    g1 = eng.step([(st.slot_of("a"), a[:100]), (st.slot_of("b"), b[:5])], "all")
    g2 = eng.step([(st.slot_of("b"), b[5:6]), (st.slot_of("a"), a[100:101])], "all")
    g3 = eng.step([(st.slot_of("a"), a[101:]), (st.slot_of("b"), b[6:])], "all")
    assert _err(torch.cat([g1[:100], g2[1:], g3[:39]]), ra) < tol and _err(torch.cat([g1[100:], g2[:1], g3[39:]]), rb) < tol


def test_pieces_cut_inside_a_step_and_the_folded_form_when_expanded_rows_would_be_too_many(monkeypatch):
    import torchao_fork_b200._models.segment_step as S
    import torchao_fork_b200._models.softmax_step as A
    for make in (_mixed, _tensor):
        cfg = make()
        w = O.random_weights(cfg, 23)
        toks = _tokens(cfg, 150, 3)
        ref = O.forward(cfg, w, toks)
        for dtype in DTYPES:
            tol = _tol(cfg, w, toks, dtype)
            for max_step, max_bytes in ((4096, 4 << 30), (37, 4 << 30), (50, 1000)):
                monkeypatch.setattr(S, "MAX_STEP_TOKENS", max_step)
                monkeypatch.setattr(A, "EXPAND_MAX_BYTES", max_bytes)
                m = _model(cfg, w, dtype)
                got = m.step_engine.step([(m.states.slot_of("a"), toks)], "all")
                assert _err(got, ref) < tol, (max_step, max_bytes, dtype)


@pytest.mark.parametrize("name", ["mixed", "odd", "tensor"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests_equal_each_alone_and_slots_are_reused(dtype, name):
    cfg = CONFIGS[name]()
    w = O.random_weights(cfg, 24)
    a, b, c = _tokens(cfg, 90, 4), _tokens(cfg, 21, 5), _tokens(cfg, 63, 6)
    ra, rb, rc = O.forward(cfg, w, a), O.forward(cfg, w, b), O.forward(cfg, w, c)
    tol = max(_tol(cfg, w, t, dtype) for t in (a, b, c))
    m = _model(cfg, w, dtype, slots=2)
    eng, st = m.step_engine, m.states
    # a prompt portion of one request beside single decoded tokens of another, request b finishes and c takes its slot
    g1 = eng.step([(st.slot_of("a"), a[:60]), (st.slot_of("b"), b[:19])], "all")
    assert _err(g1[:60], ra[:60]) < tol and _err(g1[60:], rb[:19]) < tol
    g2 = eng.step([(st.slot_of("b"), b[19:20]), (st.slot_of("a"), a[60:61])], "all")
    assert _err(g2[:1], rb[19:20]) < tol and _err(g2[1:], ra[60:61]) < tol
    g2 = eng.step([(st.slot_of("b"), b[20:]), (st.slot_of("a"), a[61:63])], "all")
    assert _err(g2[:1], rb[20:]) < tol and _err(g2[1:], ra[61:63]) < tol
    slot_b = st.slot_of("b")
    st.release("b")
    assert st.slot_of("c") == slot_b                       # the freed slot, with b's state still in it
    g3 = eng.step([(st.slot_of("a"), a[63:64]), (st.slot_of("c"), c[:61])], "all")
    assert _err(g3[:1], ra[63:64]) < tol and _err(g3[1:], rc[:61]) < tol
    g4 = eng.step([(st.slot_of("c"), c[61:]), (st.slot_of("a"), a[64:])], "all")
    assert _err(g4[:2], rc[61:]) < tol and _err(g4[2:], ra[64:]) < tol
    # a third live request makes the state manager double its slots; the old ones keep their state
    d = _tokens(cfg, 9, 7)
    g5 = eng.step([(st.slot_of("d"), d)], "all")
    assert m.max_batch_size == 4 and _err(g5, O.forward(cfg, w, d)) < max(tol, _tol(cfg, w, d, dtype))
    e = _tokens(cfg, 1, 8)
    more = eng.step([(st.slot_of("d"), e)], "all")         # ... also the last token, which the next one's embedding reads
    assert _err(more, O.forward(cfg, w, d + e)[-1:]) < max(tol, _tol(cfg, w, d + e, dtype))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_past_every_ring(dtype):
    cfg = _tensor()
    w = O.random_weights(cfg, 25)
    toks = _tokens(cfg, 170, 9)
    ref, tol = O.forward(cfg, w, toks), _tol(cfg, w, toks, dtype)
    m = _model(cfg, w, dtype, slots=1, seq=170)
    eng, st = m.step_engine, m.states
    got = [eng.step([(st.slot_of("r"), toks[:20])], "all")] + [eng.step([(st.slot_of("r"), [t])], "all") for t in toks[20:]]
    assert _err(torch.cat(got), ref) < tol
    with pytest.raises(RuntimeError):                      # the full cache has an end
        eng.step([(st.slot_of("r"), [1])], "all")
    win = O.model_config([O.attention_layer(), O.attention_layer(size=16)], loop=(0, 1, 2))      # windows only: no end
    w = O.random_weights(win, 25)
    toks = _tokens(win, 90, 9)
    m = _model(win, w, dtype, slots=1, seq=16)
    eng, st = m.step_engine, m.states
    got = [eng.step([(st.slot_of("r"), toks[:20])], "all")] + [eng.step([(st.slot_of("r"), [t])], "all") for t in toks[20:]]
    assert _err(torch.cat(got), O.forward(win, w, toks)) < _tol(win, w, toks, dtype)


def _single_out(kind, size):
    """One softmax layer whose scores single out token 1 among tokens 2 .. : the logits of a position say whether a token 1 is
    visible from it.  Token 1's embedding answers in coordinate 0; every token asks through coordinate 1."""
    W = 16
    lay = O.attention_layer(heads=1, kv_heads=1, dim=16, vdim=16, scale=8.0, size=size, rot=0, ff=0) if kind == "attention" else \
        O.latent_layer(heads=1, dim=16, rot_dim=16, vdim=16, q_rank=16, kv_rank=16, scale=8.0, ff=0)
    cfg = O.model_config([lay], width=W, vocab=24, scale=1.0, bigram=None)
    w = O.random_weights(cfg, 3)
    emb = torch.randn(24, W, generator=_gen(1))
    emb[:, 0], emb[:, 1] = 0.0, 6.0
    emb[1, 0] = 9.0
    one, ask, q = torch.zeros(16, W), torch.zeros(16, W), "l0.mix."
    one[0, 0], ask[0, 1] = 1.0, 1.0
    if kind == "attention":
        w[q + "q"], w[q + "k"], w[q + "q.norm"], w[q + "k.norm"] = ask, one, torch.ones(16), torch.ones(16)
        for s in "qkv":
            w[q + s + ".b"] = torch.zeros(16)
        w[q + "k.b"] = torch.full((16,), 1.0)               # other keys are not normed up out of nothing
    else:
        w[q + "dq"], w[q + "dq.norm"] = torch.eye(16, W), torch.ones(16)
        w[q + "uq"] = torch.cat([ask * 4, torch.zeros(16, 16)], 0)
        w[q + "dkv"], w[q + "dkv.norm"], w[q + "uk"] = torch.cat([torch.eye(16, W), torch.zeros(16, W)], 0), torch.ones(16), one
        w[q + "sink"] = torch.zeros(1)
    w["embed"], w["l0.norm1"] = emb, torch.ones(W)
    return cfg, {k: v.bfloat16() for k, v in w.items()}


@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_singled_out_token_at_the_edge_of_the_window_and_far_away(dtype, kind):
    size, at, T = 40, 30, 130
    cfg, w = _single_out(kind, size)
    toks = [2 + t % 20 for t in _tokens(cfg, T, 5)]
    toks[at] = 1
    ref = O.forward(cfg, w, toks)
    other = list(toks)
    other[at] = 2
    moved = _errs(O.forward(cfg, w, other), ref)
    tol = _tol(cfg, w, toks, dtype)
    if kind == "attention":
        assert float(moved[at + size - 1]) > 5 * tol and float(moved[at + size]) < tol / 10      # the edge shows in the oracle
    else:
        assert float(moved[T - 1]) > 5 * tol                                                     # a hundred tokens back
    for sizes in ([T], [1], [at + size, 1], [at + size - 1, 1], [2], [64, 3], [at, 37]):
        m = _model(cfg, w, dtype, slots=1)
        got = torch.cat([m.step_engine.step([(m.states.slot_of("a"), toks[a:a + c])], "all") for a, c in _cuts(T, sizes)])
        assert _err(got, ref) < tol, sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_and_the_pair_in_front_of_a_portion(dtype):
    """A sequence of one token, a portion that starts with its sequence's second token, and the same token behind different ones."""
    cfg = _mixed()
    w = O.random_weights(cfg, 31)
    m = _model(cfg, w, dtype, slots=3)
    eng, st = m.step_engine, m.states
    for i, toks in enumerate(([7], [7, 9], [8, 9], [7, 7, 7])):
        tol = _tol(cfg, w, toks, dtype)
        ref = O.forward(cfg, w, toks)
        assert _err(eng.step([(st.slot_of("w"), toks)], "all"), ref) < tol
        assert _err(torch.cat([eng.step([(st.slot_of("s"), [t])], "all") for t in toks]), ref) < tol
        st.release("w"), st.release("s")                   # the slots keep what these sequences left in them
    moved = _err(O.forward(cfg, w, [8, 9])[-1:], O.forward(cfg, w, [7, 9])[-1:])
    assert moved > 5 * _tol(cfg, w, [7, 9], dtype)


@pytest.mark.parametrize("batch", [1, 2])
def test_greedy_generation_through_generator_and_graph(batch):
    from torchao_fork_b200._models.llama.generate import Generator
    cfg = _mixed()
    w = O.random_weights(cfg, 26)
    prompt = _tokens(cfg, 13, 5)
    want = O.greedy(cfg, w, prompt, 14)
    for use_graph in (False, True):
        m = _model(cfg, w, torch.float32, slots=batch, seq=64)
        gen = Generator(m, batch, 64, temperature=0.0, top_k=None, use_graph=use_graph)
        for _ in range(2):      # the second call restarts the slots at position 0
            seq = gen.generate(torch.tensor(prompt), 14)
            assert seq.shape == (batch, 27)
            for b in range(batch):
                assert seq[b, 13:].tolist() == want, (use_graph, b)


def test_sampling_and_command_line(tmp_path):
    import importlib
    from torchao_fork_b200._models.llama.generate import Generator
    cfg = _tensor()
    w = O.random_weights(cfg, 27)
    gen = Generator(_model(cfg, w, torch.bfloat16, slots=1), 1, 60, temperature=0.8, top_k=5, use_graph=True)
    seq = gen.generate(torch.tensor(_tokens(cfg, 26, 6)), 10)
    assert seq.shape == (1, 36) and int(seq.min()) >= 0 and int(seq.max()) < cfg["vocab"]
    G = importlib.import_module("torchao_fork_b200._models.llama.generate")
    folder = str(tmp_path / "ckpt")
    O.write_checkpoint(folder, cfg, w)
    # the calls themselves are the check: folder or name -> registry -> prefill -> graph decode -> sampling
    G.main(checkpoint_path=folder, num_samples=1, max_new_tokens=9, prompt="1,2,3,4,5", temperature=0.0, precision=torch.float32)
    G.main(random_init="Sozanex-test", num_samples=1, max_new_tokens=6, prompt="7,8,9")


def test_named_configuration_through_the_registry():
    from torchao_fork_b200._models import registry
    m = registry.random_init("Sozanex-test", "cuda", torch.bfloat16)
    m.setup_caches(1, 64)
    out = m(torch.randint(0, 512, (1, 40), device="cuda"))
    assert out.shape == (1, 1, 512) and bool(torch.isfinite(out).all())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_on_a_checkpoint_folder(tmp_path, dtype):
    cfg = _mixed()
    w = O.random_weights(cfg, 28)
    folder, out = str(tmp_path / "model"), str(tmp_path / "out")
    O.write_checkpoint(folder, cfg, w)
    a, b = _tokens(cfg, 29, 7), _tokens(cfg, 12, 8)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [0, 16]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[17:19], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[19:], "want": [9]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[:11], "want": [10]}], "end": []},
             {"step": 4, "entries": [{"id": "b", "tokens": b[11:], "want": [0]}], "end": ["b"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out,
                        "--max-tokens", "64", "--slots", "1"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    assert not os.path.exists(os.path.join(out, "1.f32"))
    ra, rb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    tol = max(_tol(cfg, w, t, getattr(torch, dtype)) for t in (a, b))
    rd = lambda i: torch.from_numpy(np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    assert _err(torch.cat([rd(0), rd(2)]), ra[[0, 16, 28]]) < tol and _err(torch.cat([rd(3), rd(4)]), rb[[10, 11]]) < tol
