"""Rigalorn on the GPU against the float64 oracle (tests/rigalorn_oracle.py): every mechanism's kernel alone, then the model
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

import rigalorn_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 1e-4
F64 = torch.float64
BF16, F32 = 0, 1      # storage types of the library (AO_LM_BF16, AO_LM_F32)


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
    from torchao_fork_b200._models.rigalorn import Rigalorn, RigalornArgs
    m = Rigalorn(RigalornArgs.from_dict(cfg), w, "cuda", dtype).eval()
    m.setup_caches(slots, seq)
    return m


def _tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=_gen(seed)).tolist()


def _rows(segs):
    """[(slot, first position, rows)] -> per-row slot, pos, back, ahead and the segments' (first row, rows) on the device."""
    slot, pos, back, ahead, first, count = [], [], [], [], [], []
    for s, p0, c in segs:
        first.append(len(slot))
        count.append(c)
        slot += [s] * c
        pos += list(range(p0, p0 + c))
        back += list(range(c))
        ahead += list(range(c - 1, -1, -1))
    return _i32(slot), _i32(pos), _i32(back), _i32(ahead), _i32(first), _i32(count)


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
@pytest.mark.parametrize("W", [33, 256, 2500, 16384])
@pytest.mark.parametrize("parts", ["add_norm", "norm_rows", "add_only"])
def test_residual_add_with_rms_norm(W, parts):
    lib, L = _lm()
    n, eps = 7, 1e-5
    g = _gen(W)
    x, y = torch.randn(n, W, generator=g) * 3 + 0.5, torch.randn(n, W, generator=g)
    wt = (1 + 0.2 * torch.randn(W, generator=g)).bfloat16()
    xd, yd, wd, wf = x.cuda(), y.cuda(), wt.cuda(), wt.float().cuda()
    out = torch.zeros(n, W, device="cuda")
    if parts == "add_norm":
        lib.lm_check(L.ao_lm_add_rms_norm(_p(xd), _p(yd), None, n, W, _p(wf), F32, eps, _p(out), _st()), "norm")
        xs = x.double() + y.double()
        assert _close(xd, xs, 1e-6) and _close(out, O.rms_norm(xs, wt.double(), eps))
    elif parts == "norm_rows":
        rows = [5, 0, 3]
        rd, ob = _i32(rows), torch.zeros(3, W, device="cuda", dtype=torch.bfloat16)
        lib.lm_check(L.ao_lm_add_rms_norm(_p(xd), None, _p(rd), 3, W, _p(wd), BF16, eps, _p(ob), _st()), "norm")
        assert torch.equal(xd.cpu(), x) and _close(ob.float(), O.rms_norm(x.double()[rows], wt.double(), eps), 1e-2)
    else:
        lib.lm_check(L.ao_lm_add_rms_norm(_p(xd), _p(yd), None, n, W, None, F32, eps, None, _st()), "norm")
        assert _close(xd, x.double() + y.double(), 1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("ff,off,ld,out_off,ld_out", [(40, 8, 64, 12, 52), (37, 3, 41, 5, 43), (5000, 4, 5008, 0, 5000)])
def test_xielu_units_and_scaled_embedding(dtype, ff, off, ld, out_off, ld_out):
    lib, L = _lm()
    dt, n = (BF16 if dtype == torch.bfloat16 else F32), 5
    z = torch.randn(n, ld, generator=_gen(ff)) * 3
    z[0, off], z[1, off], z[2, off], z[3, off] = 0.0, -30.0, 1e-4, -1e-4
    p, q = torch.tensor(0.4, dtype=F64), torch.tensor(-1.3, dtype=F64)
    zd, out = z.cuda(), torch.full((n, ld_out), 9.0, device="cuda", dtype=dtype)
    lib.lm_check(L.ao_lm_xielu_rows(zd.data_ptr() + 4 * off, ld, n, ff, math.log1p(math.exp(0.4)), 0.5 + math.log1p(math.exp(-1.3)),
                                    out.data_ptr() + out.element_size() * out_off, ld_out, dt, _st()), "xielu")
    assert _close(out[:, out_off:out_off + ff].float(), O.xielu(z[:, off:off + ff].double(), p, q), 1e-6 if dt == F32 else 1e-2)
    assert float(out[:, :out_off].float().sub(9).abs().sum() + out[:, out_off + ff:].float().sub(9).abs().sum()) == 0.0
    table, tok = torch.randn(11, ff, generator=_gen(1)).to(dtype).cuda(), torch.tensor([3, 10, 0], device="cuda")
    x = torch.zeros(3, ff, device="cuda")
    lib.lm_check(L.ao_lm_embed_scaled(_p(table), dt, _p(tok), 3, ff, 0.375, _p(x), _st()), "embed")
    assert _close(x, table[tok].double() * 0.375, 1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,dims,scaling,lam", [(4, 2, 12, 8, 8, (4.0, 64, 8.0, 1.0), 0.4), (3, 1, 7, 5, 6, None, 0.0), (2, 2, 16, 16, 0, None, 1.0)])
def test_preparation_with_scaled_rotation_and_mixed_values(dtype, H, G, d, dv, dims, scaling, lam):
    from torchao_fork_b200._models.rotary import RotaryArgs
    lib, L = _lm()
    dt, n = (BF16 if dtype == torch.bfloat16 else F32), 6
    g = _gen(H + d)
    qo, ko, vo = 1, 1 + H * d, 1 + H * d + G * d
    ld = vo + G * dv + 3
    proj, pos = torch.randn(n, ld, generator=g), [0, 1, 5, 300, 301, 17]
    qb, kb, vb = (torch.randn(s, generator=g).bfloat16().to(dtype).cuda() for s in (H * d, G * d, G * dv))
    vf = torch.randn(n, G * dv, generator=g).to(dtype).cuda()
    rot = O.rotary(dims, 900.0, scaling) if dims else None
    ra = RotaryArgs.from_dict(rot)
    inv = ra.inv_freq("cuda")
    pd, posd = proj.cuda(), _i32(pos)
    qn, kn, vn = torch.zeros(n, H, d, device="cuda"), torch.zeros(n, G, d, device="cuda", dtype=dtype), torch.zeros(n, G * dv, device="cuda", dtype=dtype)
    mix = _p(vf) if lam else None
    lib.lm_check(L.ao_lm_qkv_rotary_mix_prep(_p(pd), ld, qo, ko, vo, _p(qb), _p(kb), _p(vb), _p(posd), _p(inv), dims, 1, ra.amplitude, mix, lam, n,
                                             H, G, d, G * dv, dt, _p(qn), _p(kn), _p(vn), _st()), "prep")
    p = torch.tensor(pos)
    tol = 1e-4 if dt == F32 else 1e-2
    assert _close(qn, O.rotate((proj[:, qo:ko].double() + qb.double().cpu()).view(n, H, d), p, rot, "half"), 1e-4)
    assert _close(kn.float(), O.rotate((proj[:, ko:vo].double() + kb.double().cpu()).view(n, G, d), p, rot, "half"), tol)
    v = proj[:, vo:vo + G * dv].double() + vb.double().cpu()
    assert _close(vn.float(), O.mixed_values(v, vf.double().cpu(), lam) if lam else v, tol)


def _delta_run(proj, conv_w, a_log, dt_bias, m, cuts, block=None, slots=3, slot=2, dt=F32):
    """delta_prep and delta_recurrence over one sequence cut into portions -> (qk, v, gb, read-outs [T][H][dv])."""
    lib, L = _lm()
    H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    dp, C, ld = -(-d // 4) * 4, 2 * G * d + H * dv, proj.shape[1]
    cast = (lambda t: t.cuda().bfloat16()) if dt == BF16 else (lambda t: t.cuda().float())
    cw, al, db = cast(conv_w.t().contiguous()), cast(a_log), cast(dt_bias)
    state = torch.full((slots, H, dv, dp), 7.0, device="cuda")           # a reused slot holds rubbish: position 0 must not read it
    mem = torch.full((slots, max(1, taps - 1), C), 5.0, device="cuda")
    parts = []
    for a, c in cuts:
        sd, pd, bd, _, sf, sc = _rows([(slot, a, c)])
        x = proj[a:a + c].float().cuda().contiguous()
        qk, v, gb = torch.zeros(c, 2, G, dp, device="cuda"), torch.zeros(c, H * dv, device="cuda"), torch.zeros(c, H, 2, device="cuda")
        lib.lm_check(L.ao_lm_delta_prep(_p(x), ld, 0, C, C + H, c, H, G, d, dp, dv, taps, _p(cw), _p(mem), _p(sd), _p(pd), _p(bd), _p(al), _p(db),
                                        dt, 1e-6, d ** -0.5, _p(qk), _p(v), _p(gb), _st()), "prep")
        out = torch.zeros(c, H * dv, device="cuda")
        lib.lm_check(L.ao_lm_delta_recurrence(_p(qk), _p(v), _p(gb), H, G, dp, dv, _p(state), _p(sd), _p(pd), _p(sf), _p(sc), 1,
                                              block or (1 if c == 1 else 8), _p(x), ld, C, taps, _p(mem), _p(out), _st()), "recurrence")
        parts.append((qk[..., :d], v.view(c, H, dv), gb, out.view(c, H, dv)))
    assert float(state[:slot].min()) == 7.0 and float(mem[:slot].min()) == 5.0      # other slots untouched
    return [torch.cat([p[i] for p in parts]) for i in range(4)]


def _delta_case(H, G, d, dv, taps, T=75):
    """A projection [q | k | v | a | b] of T rows, and the oracle's inputs and read-outs for it."""
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "conv": taps}
    g = _gen(H * 100 + d + taps)
    C = 2 * G * d + H * dv
    proj = torch.randn(T, C + 2 * H, generator=g)
    conv = torch.randn(C, taps, generator=g).mul(0.5).add(0.3).bfloat16()
    a_log, dt_bias = torch.randn(H, generator=g).bfloat16(), torch.randn(H, generator=g).bfloat16()
    eye = torch.eye(C + 2 * H, dtype=F64)                # the projection itself is the oracle's input row
    w = {"q": eye[:G * d], "k": eye[G * d:2 * G * d], "v": eye[2 * G * d:C], "a": eye[C:C + H], "b": eye[C + H:],
         "q.conv": conv[:G * d].double(), "k.conv": conv[G * d:2 * G * d].double(), "v.conv": conv[2 * G * d:].double(),
         "A_log": a_log.double(), "dt_bias": dt_bias.double()}
    ref = O.delta_inputs(proj.double(), w, "", m)
    return m, proj, conv, a_log, dt_bias, ref, O.delta_recurrence(*ref)


@pytest.mark.parametrize("H,G,d,dv,taps", [(2, 1, 8, 8, 4), (3, 3, 5, 7, 2), (1, 1, 12, 8, 2), (2, 2, 160, 12, 3), (3, 1, 132, 20, 2), (1, 1, 64, 40, 1), (4, 2, 30, 33, 3), (2, 2, 128, 16, 4), (6, 2, 100, 64, 5),
                                           (1, 1, 200, 9, 4), (1, 1, 300, 5, 4), (1, 1, 600, 3, 2), (2, 1, 1, 1, 7)])
def test_delta_rule_with_its_convolutions_in_portions(H, G, d, dv, taps):
    T = 75
    m, proj, conv, a_log, dt_bias, (q, k, v, g, beta), ref = _delta_case(H, G, d, dv, taps, T)
    for cuts, block in ([(0, T)], None), (_cuts(T, [1]), None), (_cuts(T, [1]), 8), (_cuts(T, [2, 17, 1, 33]), None), (_cuts(T, [2]), None), ([(0, T)], 1):
        qk, vv, gb, out = _delta_run(proj, conv, a_log, dt_bias, m, cuts, block)
        assert _close(qk[:, 0], q, 1e-5) and _close(qk[:, 1], k, 1e-5) and _close(vv, v, 1e-5), (cuts[:3], block)
        assert _close(gb[..., 0], g, 1e-5) and _close(gb[..., 1], beta, 1e-5)
        assert _close(out, ref, 3e-5), (cuts[:3], block)
    out = _delta_run(proj, conv, a_log, dt_bias, m, _cuts(T, [9, 30]), dt=BF16)[3]      # bf16 only stores the weights, which are bf16
    assert _close(out, ref, 3e-5)


def test_delta_rule_several_segments_of_unequal_length_in_one_launch():
    """Three sequences in one launch, one of them a single row that continues another launch's state."""
    lib, L = _lm()
    m, proj, conv, a_log, dt_bias, (q, k, v, g, beta), ref = _delta_case(4, 2, 12, 20, 3, 40)
    H, G, d, dv = 4, 2, 12, 20
    qk = torch.stack([q, k], 1).float().cuda()
    vd, gb = v.float().reshape(40, -1).cuda(), torch.stack([g, beta], -1).float().cuda()
    state = torch.full((4, H, dv, d), 3.0, device="cuda")
    outs = {}
    for segs, rows in (([(3, 0, 24), (1, 0, 7)], [*range(24), *range(7)]), ([(1, 7, 1), (0, 0, 2), (3, 24, 16)], [7, 0, 1, *range(24, 40)])):
        sd, pd, _, _, sf, sc = _rows(segs)
        r = torch.tensor(rows, device="cuda")
        a, b, c = qk[r].contiguous(), vd[r].contiguous(), gb[r].contiguous()
        out = torch.zeros(len(rows), H * dv, device="cuda")
        lib.lm_check(L.ao_lm_delta_recurrence(_p(a), _p(b), _p(c), H, G, d, dv, _p(state), _p(sd), _p(pd), _p(sf), _p(sc), len(segs), 8, None, 0, 0,
                                              1, None, _p(out), _st()), "recurrence")
        at = 0
        for s, p0, n in segs:
            outs.setdefault(s, []).append(out[at:at + n])
            at += n
    assert _close(torch.cat(outs[3]).view(40, H, dv), ref) and _close(torch.cat(outs[1]).view(8, H, dv), ref[:8])
    assert _close(outs[0][0].view(2, H, dv), ref[:2]) and float(state[2].min()) == 3.0


def test_delta_rule_remembers_for_hundreds_of_tokens_and_overwrites_one_key():
    """A value written under one key at position 0 is read exactly at position 399 while other keys are written in between
    (decay 1); a second write under the same key with step 1 leaves nothing of the first."""
    lib, L = _lm()
    T, d, dv = 400, 8, 4
    q, k, v = torch.zeros(T, 1, d), torch.zeros(T, 1, d), torch.randn(T, 1, dv, generator=_gen(0))
    k[:, 0, 1:] = torch.randn(T, d - 1, generator=_gen(1))
    k[0] = 0
    k[0, 0, 0] = 1.0
    k = k / k.norm(dim=-1, keepdim=True)
    q[:, 0, 0] = 1.0
    over = k.clone()
    over[200] = k[0]
    for keys, want in ((k, v[0, 0]), (over, v[200, 0])):
        for cuts in ([(0, T)], _cuts(T, [1]), _cuts(T, [129, 2, 70])):
            state, outs = torch.full((1, 1, dv, d), 3.0, device="cuda"), []
            for a, c in cuts:
                sd, pd, _, _, sf, sc = _rows([(0, a, c)])
                qk = torch.stack([q[a:a + c], keys[a:a + c]], 1).cuda()
                vd, gb, out = v[a:a + c].cuda(), torch.ones(c, 1, 2, device="cuda"), torch.zeros(c, dv, device="cuda")
                lib.lm_check(L.ao_lm_delta_recurrence(_p(qk), _p(vd), _p(gb), 1, 1, d, dv, _p(state), _p(sd), _p(pd), _p(sf), _p(sc), 1,
                                                      1 if c == 1 else 8, None, 0, 0, 1, None, _p(out), _st()), "recurrence")
                outs.append(out)
            assert _close(torch.cat(outs)[-1], want, 1e-4), cuts[:2]


@pytest.mark.parametrize("dv", [10, 700])
def test_unit_rms_per_head_with_one_weight_for_all_heads_into_a_wider_row(dv):
    lib, L = _lm()
    n, H, eps, ld = 6, 3, 1e-5, 3 * dv + 7
    g = _gen(dv)
    y, gate, wt = torch.randn(n, H * dv, generator=g) * 4, torch.randn(n, H * dv, generator=g), torch.randn(dv, generator=g).bfloat16()
    out = torch.full((n, ld), 9.0, device="cuda", dtype=torch.bfloat16)
    yd, gd, wd = y.cuda(), gate.cuda(), wt.cuda()
    lib.lm_check(L.ao_lm_gated_group_norm_rows(_p(yd), H * dv, _p(gd), H * dv, 2, n, H * dv, H, _p(wd), 1, BF16, eps, _p(out), ld, _st()), "ggn")
    ref = O.rms_norm(y.double().view(n, H, dv), wt.double(), eps).reshape(n, H * dv) * O.silu(gate.double())
    assert _close(out[:, :H * dv].float(), ref, 1e-2) and float(out[:, H * dv:].float().sub(9).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dn,dr,R,Rq,dims", [(3, 8, 4, 14, 10, 4), (2, 5, 7, 33, 100, 6), (1, 16, 16, 64, 48, 0)])
def test_latent_norms_and_rotated_parts(dtype, H, dn, dr, R, Rq, dims):
    lib, L = _lm()
    dt, n, eps = (BF16 if dtype == torch.bfloat16 else F32), 5, 1e-4
    g = _gen(R)
    ld, pos = Rq + R + dr + 5, [0, 1, 9, 700, 701]
    proj, q = torch.randn(n, ld, generator=g), torch.randn(n, H * (dn + dr), generator=g)
    wq, wc = (1 + 0.3 * torch.randn(Rq, generator=g)).bfloat16(), (1 + 0.3 * torch.randn(R, generator=g)).bfloat16()
    rot = O.rotary(dims, 700.0)
    inv = O.frequencies(rot)[0].float().cuda() if dims else None
    pd, qd, wqd, wcd, posd = proj.cuda(), q.cuda(), wq.to(dtype).cuda(), wc.to(dtype).cuda(), _i32(pos)
    cq, c, kr = (torch.zeros(n, k, device="cuda", dtype=dtype) for k in (Rq, R, dr))
    lib.lm_check(L.ao_lm_latent_low_prep(_p(pd), ld, n, 2, Rq, 2 + Rq, R, dr, _p(wqd), _p(wcd), dt, eps, dims, _p(inv), 1.0, _p(posd), _p(cq), _p(c),
                                         _p(kr), _st()), "low")
    qn, qr = torch.zeros(H, n, dn, device="cuda", dtype=dtype), torch.zeros(n, H, dr, device="cuda")
    lib.lm_check(L.ao_lm_latent_query_prep(_p(qd), n, H, dn, dr, dt, dims, _p(inv), 1.0, _p(posd), _p(qn), _p(qr), _st()), "query")
    p, x, tol = torch.tensor(pos), proj.double(), 1e-5 if dt == F32 else 1e-2
    turn = lambda t: O.rotate(t, p, rot, "interleaved") if dims else t
    assert _close(cq.float(), O.rms_norm(x[:, 2:2 + Rq], wq.double(), eps), tol)
    assert _close(c.float(), O.rms_norm(x[:, 2 + Rq:2 + Rq + R], wc.double(), eps), tol)
    assert _close(kr.float(), turn(x[:, 2 + Rq + R:2 + Rq + R + dr].reshape(n, 1, dr)).view(n, dr), max(tol, 1e-4))
    qq = q.double().view(n, H, dn + dr)
    assert _close(qn.float(), qq[..., :dn].transpose(0, 1), tol) and _close(qr, turn(qq[..., dn:].contiguous()), 1e-4)


def _latent_run(qn, qr, c, kr, uk, uv, cuts, window, scale, ring, dtype, form, n_split=1, slot=1, slots=3, ld_pad=0):
    """Latent attention under a window over one sequence cut into portions; qn [T][H][dn], qr [T][H][dr], c [T][R], kr [T][dr],
    uk [H][dn][R], uv [H][dv][R].  form "folded": -> weighted latents [T][H][R]; "expanded": -> heads [T][H][dv]."""
    lib, L = _lm()
    T, H, dn = qn.shape
    dr, R, dv = qr.shape[-1], c.shape[-1], uv.shape[1]
    dt = BF16 if dtype == torch.bfloat16 else F32
    rows = ctypes.c_int()
    plan = L.ao_lm_latent_attention_plan(dt, H, R, dr, ctypes.byref(rows)) if form == "folded" else \
        L.ao_lm_latent_attention_expanded_plan(dt, dn, dr, dv, ctypes.byref(rows))
    lib.lm_check(plan, "plan")
    assert rows.value > 0
    rc, rk = (torch.full((slots, ring, k), 50.0, device="cuda", dtype=dtype) for k in (R, dr))   # rubbish that must not be seen
    outs = []
    for a, n in cuts:
        segs = [(slot, a, n)]
        sd, pd, bd, ad, _, _ = _rows(segs)
        tf, tc = _tiles(segs, rows.value)
        cd, kd = c[a:a + n].to(dtype).cuda().contiguous(), kr[a:a + n].to(dtype).cuda().contiguous()
        qrd = qr[a:a + n].float().cuda().contiguous()
        if form == "folded":
            qa = torch.einsum("thd,hdr->htr", qn[a:a + n], uk).float().cuda().contiguous()
            ws = torch.zeros(max(16, int(L.ao_lm_latent_attention_workspace_bytes(n, H, R, n_split))), dtype=torch.uint8, device="cuda")
            ws.view(torch.float32)[:] = float("nan")         # shares that see no key must not be read
            out = torch.zeros(n, H, R, device="cuda", dtype=dtype)
            lib.lm_check(L.ao_lm_window_latent_attention(_p(qa), _p(qrd), _p(rc), _p(rk), _p(cd), _p(kd), dt, ring, _p(sd), _p(pd), _p(bd), _p(tf),
                                                         _p(tc), len(tf), n, H, R, dr, scale, window, None, None, n_split, _p(ws), ws.numel(),
                                                         _p(out), _st()), "folded")
            outs.append(out.float())
        else:
            h = min(a, window - 1)
            src = _i32([-1 - (slot * ring + p % ring) for p in range(a - h, a)] + list(range(n)))
            ca, ka = torch.zeros(h + n, R, device="cuda", dtype=dtype), torch.zeros(h + n, dr, device="cuda", dtype=dtype)
            lib.lm_check(L.ao_lm_latent_rows_gather(_p(src), h + n, _p(cd), _p(kd), _p(rc), _p(rk), dt, R, dr, _p(ca), _p(ka), _st()), "gather")
            assert torch.equal(ca.cpu().double(), c[a - h:a + n].to(dtype).double()) and torch.equal(ka.cpu().double(), kr[a - h:a + n].to(dtype).double())
            kv = torch.cat([torch.einsum("tr,hdr->thd", ca.double(), uk.cuda()).flatten(1), torch.einsum("tr,hdr->thd", ca.double(), uv.cuda()).flatten(1)], 1)
            kv = kv.to(dtype).contiguous()
            ld, ldo = H * (dn + dv), H * dv + ld_pad
            qd, k0 = qn[a:a + n].transpose(0, 1).to(dtype).cuda().contiguous(), _i32([h - a] * len(tf))
            out = torch.zeros(n, ldo, device="cuda", dtype=dtype)
            lib.lm_check(L.ao_lm_window_latent_attention_expanded(_p(qd), _p(qrd), _p(kv), ld, kv.data_ptr() + kv.element_size() * H * dn, ld, _p(ka),
                                                                  dt, _p(pd), _p(tf), _p(tc), _p(k0), len(tf), n, H, dn, dr, dv, scale, window,
                                                                  None, None, _p(out), ldo, _st()), "expanded")
            outs.append(out[:, :H * dv].reshape(n, H, dv).float())
        lib.lm_check(L.ao_lm_ring_append(_p(cd), _p(kd), n, R, dr, ring, dt, _p(sd), _p(pd), _p(ad), _p(rc), _p(rk), _st()), "append")
    assert float(rc[:slot].float().min()) == 50.0
    return torch.cat(outs)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dn,dr,R,window", [(3, 8, 4, 14, 9), (1, 5, 3, 33, 1), (6, 16, 16, 64, 20), (16, 8, 16, 128, 40), (20, 4, 32, 64, 70), (5, 4, 8, 500, 13)])
def test_latent_attention_under_a_window_folded_form(dtype, H, dn, dr, R, window):
    T, scale, dv = 90, 0.3, 4
    g = _gen(H + R)
    rnd = lambda *s: torch.randn(*s, generator=g).bfloat16().double()
    qn, qr, c, kr = rnd(T, H, dn), rnd(T, H, dr), rnd(T, R), rnd(T, dr)
    uk, uv = rnd(H, dn, R) / math.sqrt(R), rnd(H, dv, R)
    qa = torch.einsum("thd,hdr->thr", qn, uk)
    ref = O.window_softmax(torch.cat([qa, qr], -1), torch.cat([c, kr], -1)[:, None], c[:, None], scale, window)
    tol = 1e-4 if dtype == torch.float32 else 2e-2
    for cuts, ring, ns in (([(0, T)], window, 1), (_cuts(T, [1]), window, 1), (_cuts(T, [2, 7, 1, 19]), window + 3, 1), (_cuts(T, [1]), window, 2),
                           (_cuts(T, [25, 1, 1]), window + 40, 3), ([(0, T)], window, 64)):
        assert _close(_latent_run(qn, qr, c, kr, uk, uv, cuts, window, scale, ring, dtype, "folded", ns), ref, tol), (cuts[:3], ring, ns)


@pytest.mark.parametrize("H,dn,dr,dv,R,window", [(2, 16, 16, 32, 24, 9), (1, 32, 16, 48, 40, 1), (3, 64, 32, 128, 16, 70), (2, 16, 48, 16, 8, 1000)])
def test_latent_attention_under_a_window_expanded_form(H, dn, dr, dv, R, window):
    T, scale = 210, 0.3
    g = _gen(H + R)
    rnd = lambda *s: torch.randn(*s, generator=g).bfloat16().double()
    qn, qr, c, kr, uk, uv = rnd(T, H, dn), rnd(T, H, dr), rnd(T, R), rnd(T, dr), rnd(H, dn, R) / 4, rnd(H, dv, R)
    k, v = (torch.einsum("tr,hdr->thd", c, u).bfloat16().double() for u in (uk, uv))
    ref = O.window_softmax(torch.cat([qn, qr], -1), torch.cat([k, kr[:, None].expand(T, H, dr)], -1), v, scale, window)
    for cuts, ring, pad in (([(0, T)], window, 0), (_cuts(T, [64, 1, 70, 17]), window + 5, 3), (_cuts(T, [130, 3]), window + 100, 8), (_cuts(T, [2]), window, 0)):
        assert _close(_latent_run(qn, qr, c, kr, uk, uv, cuts, window, scale, ring, torch.bfloat16, "expanded", ld_pad=pad), ref, 1e-2), (cuts[:3], ring)


@pytest.mark.parametrize("form,dtype", [("folded", torch.float32), ("folded", torch.bfloat16), ("expanded", torch.bfloat16)])
@pytest.mark.parametrize("how", ["whole", "portions", "decoded"])
@pytest.mark.parametrize("part", ["latent", "rotated"])
def test_one_dominant_latent_row_just_inside_and_just_outside_the_window(form, dtype, how, part):
    """Window 40.  One row answers one query so strongly that the query returns that row's values where the window lets it see
    them; one step further out, or in the future, it must leave no trace."""
    T, H, dn, dr, dv, R, window, query = 151, 2, 16, 16, 16, 64, 40, 99
    g = _gen(7)
    c = torch.randn(T, R, generator=g).bfloat16().double()
    c[:, 0] = 0
    uk, uv = torch.zeros(H, dn, R, dtype=F64), torch.randn(H, dv, R, generator=g).bfloat16().double() / 8
    uk[:, 0, 0], uv[:, :, 0] = 1.0, 0.0
    cuts = {"whole": [(0, T)], "portions": _cuts(T, [37, 2, 5]), "decoded": [(0, 38)] + [(i, 1) for i in range(38, T)]}[how]
    for key, seen in ((60, True), (59, False), (99, True), (98, True), (100, False), (64, True), (0, False)):
        qn, qr, kr, cc = torch.zeros(T, H, dn, dtype=F64), torch.zeros(T, H, dr, dtype=F64), torch.zeros(T, dr, dtype=F64), c.clone()
        if part == "latent":
            qn[query, :, 0], cc[key, 0] = 32.0, 32.0
        else:
            qr[query, :, 3], kr[key, 3] = 32.0, 32.0
        got = _latent_run(qn, qr, cc, kr, uk, uv, cuts, window, 1.0, 45, dtype, form, 3 if how == "decoded" and form == "folded" else 1)[query, 1]
        val = cc if form == "folded" else cc @ uv[1].T
        want = val[key] if seen else val[max(0, query - window + 1):query + 1].mean(0)
        assert _close(got, want, 1e-4 if dtype == torch.float32 else 2e-2), key


# ------------------------------------------------------------------------------------------------ the model
def _mixed():     # every mixer twice, value mixing with a plain attention layer between, one layer without feed-forward
    return O.model_config([O.latent_layer(), O.attention_layer(v_mix=True, scaling=(4.0, 24, 4.0, 1.0)), O.delta_layer(),
                           O.attention_layer(heads=2, kv_heads=1, dim=6, vdim=10, size=5, rot=6), O.delta_layer(heads=3, kv_heads=3, conv=4, ff=0),
                           O.attention_layer(v_mix=True, heads=2, kv_heads=2, size=13, rot=12), O.latent_layer(heads=2, size=6, ff=24)])


def _ones():      # sizes that are 1 or equal, windows of one token
    return O.model_config([O.attention_layer(heads=1, kv_heads=1, dim=16, vdim=16, size=1, rot=16, v_mix=True, ff=16),
                           O.latent_layer(heads=1, dim=16, rot_dim=16, vdim=16, q_rank=16, kv_rank=16, size=1, ff=16),
                           O.delta_layer(heads=1, kv_heads=1, dim=16, vdim=16, conv=1, ff=16),
                           O.attention_layer(heads=1, kv_heads=1, dim=16, vdim=16, size=16, rot=16, v_mix=True, ff=16)], width=16, vocab=16, scale=1.0)


def _odd():       # odd sizes everywhere
    return O.model_config([O.delta_layer(heads=3, kv_heads=1, dim=5, vdim=7, conv=5, ff=29), O.latent_layer(heads=5, dim=3, rot_dim=6, vdim=9, q_rank=7, kv_rank=11, size=7, ff=9),
                           O.attention_layer(heads=3, kv_heads=1, dim=5, vdim=7, size=3, rot=2, scaling=(2.0, 9, 1.5, 1.2), ff=0)], width=27, vocab=31, eps=1e-3, scale=2.5)


def _wide():      # windows that no test sequence outgrows or that are absent, head shapes that the tensor-core kernels cover
    return O.model_config([O.latent_layer(heads=4, dim=32, rot_dim=16, vdim=48, q_rank=24, kv_rank=64, size=1000, ff=64),
                           O.attention_layer(heads=4, kv_heads=1, dim=32, vdim=64, size=0, rot=32, scale=0.2, v_mix=True, ff=64),
                           O.delta_layer(heads=2, kv_heads=1, dim=64, vdim=32, conv=4, ff=48),
                           O.attention_layer(heads=2, kv_heads=2, dim=16, vdim=32, size=0, rot=0, v_mix=True, ff=0)], width=64, vocab=97)


def _tensor():    # the same head shapes under windows that prompts outgrow
    cfg = _wide()
    cfg["layers"][0]["mixer"]["mask"] = {"size": 50}
    cfg["layers"][1]["mixer"]["mask"] = {"size": 33}
    return cfg


CONFIGS = {"mixed": _mixed, "ones": _ones, "odd": _odd, "wide": _wide, "tensor": _tensor}
DTYPES = [torch.float32, torch.bfloat16]


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompt_and_every_layer_against_oracle(name, dtype):
    cfg = CONFIGS[name]()
    w = O.random_weights(cfg, 21)
    toks = _tokens(cfg, 45, 1)
    layers = []
    ref = O.forward(cfg, w, toks, layers_out=layers)
    m = _model(cfg, w, dtype)
    logits, sums = m.step_engine.layer_sums(m.states.slot_of("a"), toks)
    assert _err(logits, ref) < _tol(cfg, w, toks, dtype)
    if dtype == torch.float32:
        assert sums.shape[0] == len(layers)
        for r in range(sums.shape[0]):
            assert _close(sums[r], layers[r], 1e-4), r


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_prefill_equals_token_by_token_and_portions(dtype, name):
    cfg = CONFIGS[name]()
    w = O.random_weights(cfg, 22)
    toks = _tokens(cfg, 70, 2)
    ref, tol = O.forward(cfg, w, toks), 0
    tol = _tol(cfg, w, toks, dtype)
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
    import torchao_fork_b200._models.softmax_step as RS
    import torchao_fork_b200._models.segment_step as S
    for make in (_mixed, _tensor):
        cfg = make()
        w = O.random_weights(cfg, 23)
        toks = _tokens(cfg, 150, 3)
        ref = O.forward(cfg, w, toks)
        for dtype in DTYPES:
            tol = _tol(cfg, w, toks, dtype)
            for max_step, max_bytes in ((4096, 4 << 30), (37, 4 << 30), (50, 1000)):
                monkeypatch.setattr(S, "MAX_STEP_TOKENS", max_step)
                monkeypatch.setattr(RS, "EXPAND_MAX_BYTES", max_bytes)
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
    g1 = eng.step([(st.slot_of("a"), a[:60]), (st.slot_of("b"), b[:20])], "all")
    assert _err(g1[:60], ra[:60]) < tol and _err(g1[60:], rb[:20]) < tol
    g2 = eng.step([(st.slot_of("b"), b[20:]), (st.slot_of("a"), a[60:63])], "all")
    assert _err(g2[:1], rb[20:]) < tol and _err(g2[1:], ra[60:63]) < tol
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


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_past_every_ring(dtype):
    cfg = _mixed()
    w = O.random_weights(cfg, 25)
    toks = _tokens(cfg, 150, 9)
    ref, tol = O.forward(cfg, w, toks), _tol(cfg, w, toks, dtype)
    m = _model(cfg, w, dtype, slots=1, seq=64)        # every window fits 64 positions: the sequence may outgrow them
    eng, st = m.step_engine, m.states
    got = [eng.step([(st.slot_of("r"), toks[:20])], "all")] + [eng.step([(st.slot_of("r"), [t])], "all") for t in toks[20:]]
    assert _err(torch.cat(got), ref) < tol
    wide = _wide()
    m = _model(wide, O.random_weights(wide, 25), dtype, slots=1, seq=50)      # windows were cut to the cache: it has an end
    m.step_engine.step([(m.states.slot_of("r"), _tokens(wide, 50, 1))], "last")
    with pytest.raises(RuntimeError):
        m.step_engine.step([(m.states.slot_of("r"), [1])], "all")


def _edge_model(kind, size):
    """One softmax layer whose scores single out token 1 among tokens 2 .. : the logits of a position say whether a token 1 lies
    inside its window."""
    W = 16
    mk = O.attention_layer if kind == "attention" else O.latent_layer
    lay = mk(heads=1, kv_heads=1, dim=16, vdim=16, scale=1.0, size=size, rot=0, ff=0) if kind == "attention" else \
        mk(heads=1, dim=16, rot_dim=16, vdim=16, q_rank=16, kv_rank=16, scale=1.0, size=size, ff=0)
    cfg = O.model_config([lay], width=W, vocab=24, scale=1.0)
    w = O.random_weights(cfg, 3)
    one = torch.zeros(16, W)
    one[0, 0] = 1.0
    emb = torch.randn(24, W, generator=_gen(1))
    emb[:, 0], emb[:, 1] = 0.0, 4.0                      # coordinate 1: every token asks; coordinate 0: only token 1 answers
    emb[1, 0] = 4.0
    ask = torch.zeros(16, W)
    ask[0, 1] = 30.0
    q = "l0.mix."
    if kind == "attention":
        w[q + "q"], w[q + "k"] = ask, one
        for s in "qkv":
            w[q + s + ".b"] = torch.zeros(16)
    else:
        w[q + "dq"], w[q + "dq.norm"] = torch.eye(16, W), torch.ones(16)
        w[q + "uq"] = torch.cat([ask, torch.zeros(16, 16)], 0)
        w[q + "dkv"], w[q + "dkv.norm"], w[q + "uk"] = torch.cat([torch.eye(16, W), torch.zeros(16, W)], 0), torch.ones(16), one
    w["embed"], w["l0.norm1"] = emb, torch.ones(W)
    return cfg, {k: v.bfloat16() for k, v in w.items()}


@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_singled_out_token_at_the_edge_of_the_window_in_prompts_and_decoding(dtype, kind):
    size, at, T = 40, 30, 110
    cfg, w = _edge_model(kind, size)
    toks = [2 + t % 20 for t in _tokens(cfg, T, 5)]
    toks[at] = 1
    ref = O.forward(cfg, w, toks)
    other = list(toks)
    other[at] = 2
    gone = O.forward(cfg, w, other)
    tol = _tol(cfg, w, toks, dtype)
    moved = _errs(gone, ref)
    assert float(moved[at + size - 1]) > 10 * tol and float(moved[at + size]) < tol / 10      # the edge shows in the oracle
    for sizes in ([T], [1], [at + size, 1], [at + size - 1, 1], [2], [64, 3], [at, 37]):
        m = _model(cfg, w, dtype, slots=1)
        got = torch.cat([m.step_engine.step([(m.states.slot_of("a"), toks[a:a + c])], "all") for a, c in _cuts(T, sizes)])
        assert _err(got, ref) < tol, sizes


@pytest.mark.parametrize("batch", [1, 2])
def test_greedy_generation_through_generator_and_graph(batch):
    from torchao_fork_b200._models.llama.generate import Generator
    cfg = _mixed()
    w = O.random_weights(cfg, 26)
    prompt = _tokens(cfg, 13, 5)
    want = O.greedy(cfg, w, prompt, 14)
    for use_graph in (False, True):
        m = _model(cfg, w, torch.float32, slots=batch)
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
    G.main(random_init="Rigalorn-test", num_samples=1, max_new_tokens=6, prompt="7,8,9")


def test_named_configuration_through_the_registry():
    from torchao_fork_b200._models import registry
    m = registry.random_init("Rigalorn-test", "cuda", torch.bfloat16)
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
