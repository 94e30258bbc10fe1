"""Prefill and decode throughput of Rigalorn layers at sizes of real models (random weights), beside the framework's closest
existing family — Fedipel, which also mixes softmax attention under a sliding window with matrix-state recurrences — at
equal size in bf16 (the named configurations of the same width, layer count, vocabulary and feed-forward weights), and the
design's own kernels timed alone against their roofline, each beside the like kernel of an existing family.
`python bench.py --workload rigalorn-layers` prints the result as one JSON line; this file is the measurement.

Timing: CUDA events on the launching stream after 3 warm-up runs; model inputs and weights exceed L2, the kernel-alone
timings write a 256 MB buffer between runs.  Rooflines: measured copy bandwidth and cuBLAS bf16 rate of
MEASURED_PEAKS.json ("of measured"), or 6.65 TB/s and 1590 TF/s ("of fallback"); the fp32 multiply-add rate that the
matrix-state recurrences are held to is 148 SMs x 128 lanes x 2 x 1.9 GHz = 72 TF/s (nominal).
"""
import ctypes
import json
import os
import sys

import numpy as np
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

from benchmarks.bitipel_bench import peaks, timed  # noqa: E402

FP32_TFLOPS = 148 * 128 * 2 * 1.9e9 / 1e12
BF16, F32 = 0, 1


def model_numbers(names, prompt_len, decode_ctx, decode_steps, make=None):
    """prefill tokens/s of a prompt and decode tokens/s (batch 1, CUDA graph) for every named configuration; make: name -> a
    function that builds the model, for configurations that the registry does not name."""
    from torchao_fork_b200._models import registry
    from torchao_fork_b200._models.llama.generate import Generator, prefill
    dev = torch.device("cuda")
    out = {}
    for nm in names:
        model = make[nm]() if make and nm in make else registry.random_init(nm, dev, torch.bfloat16)
        S = max(prompt_len, decode_ctx + decode_steps + 8)
        gen = Generator(model, 1, S, temperature=0.0, top_k=None)
        prompt = torch.randint(0, model.config.vocab_size, (1, prompt_len), device=dev)
        pos = torch.arange(prompt_len, device=dev, dtype=torch.int32)
        with torch.no_grad():
            ms_prefill = timed(lambda: prefill(model, prompt, pos, temperature=0.0, top_k=None), iters=8, warmup=3)
            prefill(model, prompt[:, :decode_ctx], pos[:decode_ctx], temperature=0.0, top_k=None)

            def decode():
                gen.engine.set_state(torch.zeros(1, dtype=torch.int64, device=dev), decode_ctx)
                gen.decode_tokens(decode_steps)
            ms_decode = timed(decode, iters=3, warmup=2) / decode_steps
        wb = model.weight_bytes(True)
        out[nm] = {"prefill_tokens": prompt_len, "prefill_ms": round(ms_prefill, 3),
                   "prefill_tok_per_s": round(prompt_len / ms_prefill * 1e3, 1), "decode_context": decode_ctx,
                   "decode_ms_per_token": round(ms_decode, 4), "decode_tok_per_s": round(1e3 / ms_decode, 1),
                   "decode_weight_gbs": round(wb / ms_decode / 1e6, 1),
                   "launches_per_decode_step": int(getattr(gen.engine, "launches_per_step", 0)), "weight_gb": round(wb / 1e9, 3),
                   "state_bytes_per_sequence": model.state_bytes_per_sequence()}
        del gen, model
        torch.cuda.empty_cache()
    return out


class Bench:
    """Kernels alone at one configuration's layer shapes."""

    def __init__(self, name, prompt_len, decode_ctx):
        from torchao_fork_b200._models.rigalorn import rigalorn_configs
        self.setup(rigalorn_configs[name](), prompt_len, decode_ctx)
        self.delta = self.by["delta"].mixer

    def setup(self, cfg, prompt_len, decode_ctx):
        from torchao_fork_b200 import _lib
        self.lib, self.L = _lib, _lib.lm()
        self.hbm, self.tf, self.src = peaks()
        self.dev = torch.device("cuda")
        self.st = torch.cuda.current_stream().cuda_stream
        self.cfg = cfg
        self.by = {la.type: la for la in cfg.layers}
        self.att, self.lat = self.by["attention"].mixer, self.by["latent_attention"].mixer
        self.ff, self.W, self.n, self.ctx = self.cfg.layers[0].ff, self.cfg.width, prompt_len, decode_ctx
        self.flush = torch.zeros(64 << 20, dtype=torch.float32, device=self.dev)
        pos = np.arange(prompt_len)
        self.slot, self.pos, self.back = self.i32(pos * 0), self.i32(pos), self.i32(pos)
        self.one, self.last, self.zero = self.i32([1]), self.i32([decode_ctx]), self.i32([0])
        self.res = {"roofline_source": self.src, "hbm_gbs": self.hbm, "bf16_tflops": self.tf, "fp32_fma_tflops_nominal": round(FP32_TFLOPS, 1)}

    def i32(self, v):
        return torch.as_tensor(np.asarray(v, np.int32)).to(self.dev)

    def bf(self, *s):
        return torch.randn(*s, dtype=torch.bfloat16, device=self.dev)

    def f32(self, *s):
        return torch.randn(*s, dtype=torch.float32, device=self.dev)

    def tiles(self, rows):
        first = np.arange(0, self.n, rows)
        return self.i32(first), self.i32(np.minimum(rows, self.n - first)), len(first)

    def call(self, fn, *args):
        """Times one entry point; tensors are passed as their pointers (and stay referenced while it runs)."""
        raw = [a.data_ptr() if isinstance(a, torch.Tensor) else a for a in args]
        f = getattr(self.L, "ao_lm_" + fn)
        return timed(lambda: self.lib.lm_check(f(*raw, self.st), fn), flush=self.flush)

    def bytes_row(self, key, ms, byts, **more):
        self.res[key] = {"us": round(ms * 1e3, 2), "gbs": round(byts / ms / 1e6, 1), "frac_hbm": round(byts / ms / 1e6 / self.hbm, 4), **more}

    def tensor_row(self, key, ms, flops, issued):
        self.res[key] = {"ms": round(ms, 4), "tflops": round(flops / ms / 1e9, 2), "frac_bf16_tensor_peak": round(flops / ms / 1e9 / self.tf, 4),
                         "issued_tflops": round(issued / ms / 1e9, 2), "frac_issued": round(issued / ms / 1e9 / self.tf, 4)}

    # ------------------------------------------------------------------------------------------------ latent attention
    def latent(self):
        a, n, L = self.lat, self.n, self.L
        H, dn, dr, dv, R, Rq = a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank
        qn, qr, kr = self.bf(H, n, dn), self.f32(n, H, dr), self.bf(n, dr)
        kx, vx, out = self.bf(n, H * dn), self.bf(n, H * dv), self.bf(n, H * dv)
        kv, ld = torch.cat([kx, vx], 1), H * (dn + dv)
        sink, gate = self.bf(H), torch.ones(n, H, dtype=torch.float32, device=self.dev)
        rows = ctypes.c_int()
        L.ao_lm_latent_attention_expanded_plan(BF16, dn, dr, dv, ctypes.byref(rows))
        tf, tc, nt = self.tiles(rows.value)
        key0 = self.i32(np.zeros(nt))
        for key, window in (("latent_prompt", n), ("latent_prompt_window_512", 512)):
            i = np.arange(n)
            pairs = float(np.minimum(i + 1, window).sum())
            flops, issued = 2.0 * pairs * H * (dn + dr + dv), 2.0 * pairs * H * (dn + 2 * dr + 3 * dv)
            ms = self.call("window_latent_attention_expanded", qn, qr, kv, ld, kv.data_ptr() + 2 * H * dn, ld, kr, BF16, self.pos, tf, tc, key0, nt, n,
                           H, dn, dr, dv, a.scale, window, None, None, out, H * dv)
            self.tensor_row(key, ms, flops, issued)
        pairs = n * (n + 1) / 2
        ms = self.call("latent_attention_expanded", qn, qr, kx, vx, kr, BF16, n, self.slot, self.pos, tf, tc, key0, nt, n, H, dn, dr, dv, a.scale, sink,
                       gate, out)
        self.tensor_row("bitipel_latent_prompt", ms, 2.0 * pairs * H * (dn + dr + dv), 2.0 * pairs * H * (dn + 2 * dr + 3 * dv))
        # one decoded token over the cached latents, key splits as the step function picks them
        S, ctx = self.ctx + 64, self.ctx
        ring_c, ring_kr, c1, kr1 = self.bf(1, S, R), self.bf(1, S, dr), self.bf(1, R), self.bf(1, dr)
        qa, qr1, olat = self.f32(H, 1, R), self.f32(1, H, dr), self.bf(1, H, R)
        ns = max(1, min(-(-S // 32), -(-4 * 148 // -(-H // 16)), 64))
        ws = torch.zeros(int(L.ao_lm_latent_attention_workspace_bytes(1, H, R, ns)), dtype=torch.uint8, device=self.dev)
        byts = ctx * (R + dr) * 2
        ms = self.call("window_latent_attention", qa, qr1, ring_c, ring_kr, c1, kr1, BF16, S, self.zero, self.last, self.zero, self.zero, self.one, 1, 1, H,
                       R, dr, a.scale, S, None, None, ns, ws, ws.numel(), olat)
        self.bytes_row("latent_decode", ms, byts, splits=ns)
        ns2 = max(1, min(-(-S // 32), -(-2 * 148 // -(-H // 16)), 64))
        ms = self.call("latent_attention", qa, qr1, ring_c, ring_kr, BF16, S, self.zero, self.last, self.zero, self.one, 1, 1, H, R, dr, a.scale, sink,
                       gate, S - 1, ns2, ws, ws.numel(), olat)
        self.bytes_row("bitipel_latent_decode", ms, byts, splits=ns2)
        # row kernels around it
        ldp = Rq + R + dr
        proj, wq, wc, inv = self.f32(n, ldp), self.bf(Rq), self.bf(R), a.rot.inv_freq(self.dev)
        cq, c, krr = self.bf(n, Rq), self.bf(n, R), self.bf(n, dr)
        ms = self.call("latent_low_prep", proj, ldp, n, 0, Rq, Rq, R, dr, wq, wc, BF16, 1e-6, a.rot.dims, inv, 1.0, self.pos, cq, c, krr)
        self.bytes_row("latent_low_prep", ms, n * ldp * 6)
        q = self.f32(n, H * (dn + dr))
        ms = self.call("latent_query_prep", q, n, H, dn, dr, BF16, a.rot.dims, inv, 1.0, self.pos, qn, qr)
        self.bytes_row("latent_query_prep", ms, n * H * (dn * 6 + dr * 8))
        ldb = H * (dn + dr) + R + dr + H
        pb, cc, kc = self.bf(n, ldb), self.bf(1, n, R), self.bf(1, n, dr)
        ms = self.call("latent_prep", pb, BF16, ldb, n, H, dn, dr, R, 0, H * (dn + dr), H * (dn + dr) + R + dr, wc, 1e-6, a.rot.dims, inv, self.slot,
                       self.pos, cc, kc, n, qn, qr, gate)
        self.bytes_row("bitipel_latent_prep", ms, n * (ldb * 2 + H * dn * 2 + H * dr * 4 + (R + dr) * 2))

    # ------------------------------------------------------------------------------------------------ window attention
    def attention(self):
        a, n, L = self.att, self.n, self.L
        H, G, d, dv = a.heads, a.kv_heads, a.dim, a.vdim
        C = self.ctx + 64
        qn, kn, vn, out = self.f32(n, H, d), self.bf(n, G, d), self.bf(n, G, dv), self.bf(n, H * dv)
        rk, rv = self.bf(1, max(C, n), G * d), self.bf(1, max(C, n), G * dv)
        rows = ctypes.c_int()
        pairs = n * (n + 1) / 2
        L.ao_lm_window_attention_prompt_plan(BF16, 1, H, G, d, dv, ctypes.byref(rows))
        tf, tc, nt = self.tiles(rows.value)
        ms = self.call("window_attention_prompt", qn, kn, vn, rk, rv, None, None, n, 0, BF16, self.slot, self.pos, self.back, tf, tc, nt, 1, H, G, d, dv, n, 0,
                       a.scale, 0.0, 0, 0.0, 1.0, out, H * dv)
        self.tensor_row("window_prompt_one_map", ms, 2.0 * pairs * H * (d + dv), 2.0 * pairs * H * (d + 3 * dv))
        q2, k2, rk2 = self.f32(n, H, 2, d // 2), self.bf(n, G, 2, d // 2), self.bf(1, n, G * d)
        L.ao_lm_window_attention_prompt_plan(BF16, 2, H, G, d // 2, dv, ctypes.byref(rows))
        tf, tc, nt = self.tiles(rows.value)
        ms = self.call("window_attention_prompt", q2, k2, vn, rk2, rv, None, None, n, 0, BF16, self.slot, self.pos, self.back, tf, tc, nt, 2, H, G, d // 2, dv, n,
                       0, a.scale, 0.5, 1, 1e-6, 1.0, out, H * dv)
        self.tensor_row("fedipel_window_prompt_two_maps", ms, 4.0 * pairs * H * (d // 2 + dv), 4.0 * pairs * H * (d // 2 + 3 * dv))
        for key, maps, dd in (("window_decode_one_map", 1, d), ("fedipel_window_decode_two_maps", 2, d // 2)):
            ns = max(1, min(-(-C // 32), -(-4 * 148 // G), 64))
            ws = torch.zeros(int(L.ao_lm_window_attention_workspace_bytes(1, maps, H, G, dv, ns)), dtype=torch.uint8, device=self.dev)
            ms = self.call("window_attention", qn, kn, vn, rk, rv, None, None, C, 0, BF16, self.zero, self.last, self.zero, self.zero, self.one, 1, maps, H, G, dd, dv,
                           C, 0, a.scale, 0.5, maps - 1, 1e-6, 1.0, ns, ws, ws.numel(), out, H * dv)
            self.bytes_row(key, ms, self.ctx * G * (d + dv) * 2, splits=ns)
        ld = H * d + G * d + G * dv + self.ff
        proj, qb, kb, vb, vf = self.f32(n, ld), self.bf(H * d), self.bf(G * d), self.bf(G * dv), self.bf(n, G * dv)
        inv = a.rot.inv_freq(self.dev)
        byts = n * ((H * d + G * (d + dv)) * 4 + H * d * 4 + G * (d + dv) * 2)
        ms = self.call("qkv_rotary_mix_prep", proj, ld, 0, H * d, H * d + G * d, qb, kb, vb, self.pos, inv, a.rot.dims, 1, 1.2, vf, 0.3, n, H, G, d, G * dv, BF16, qn,
                       kn, vn)
        self.bytes_row("qkv_rotary_mix_prep", ms, byts + n * G * dv * 2)
        ms = self.call("qkv_rotary_prep", proj, ld, 0, H * d, H * d + G * d, qb, kb, vb, self.pos, inv, a.rot.dims, 1, n, H, G, d, G * dv, BF16, qn, kn, vn)
        self.bytes_row("fedipel_qkv_rotary_prep", ms, byts)

    # ------------------------------------------------------------------------------------------------ gated delta rule
    def recurrence(self):
        from torchao_fork_b200._models.segment_step import REC_TILE, scan_tiles
        a, n, L = self.delta, self.n, self.L
        H, G, d, dv, taps, C = a.heads, a.kv_heads, a.dim, a.vdim, a.taps, a.channels
        dp, ld = a.padded_dim, C + H * dv + self.ff + 2 * H
        proj, cw, mem = self.f32(n, ld), self.bf(taps, C), self.f32(1, taps - 1, C)
        al, db = self.bf(H), self.bf(H)
        qk, v, gb, state, out = self.f32(n, 2, G, dp), self.f32(n, H * dv), torch.rand(n, H, 2, device=self.dev), self.f32(1, H, dv, dp), self.f32(n, H * dv)
        qk /= qk.norm(dim=-1, keepdim=True)
        b_off = ld - H
        prep = lambda rows, pos: self.call("delta_prep", proj, ld, 0, b_off - H, b_off, rows, H, G, d, dp, dv, taps, cw, mem, self.slot, pos, self.back, al, db, BF16,
                                           1e-6, d ** -0.5, qk, v, gb)
        ms = prep(n, self.pos)
        self.bytes_row("delta_prep", ms, n * (C + 2 * H) * 8)
        sq, sa, sb = self.f32(n, C), self.f32(n, H), self.f32(n, H)
        ms = self.call("ssd_prep", proj, ld, 0, b_off, n, C, taps, cw, None, BF16, mem, self.slot, self.pos, self.back, H, db, al, sq, sa, sb)
        self.bytes_row("rutusun_ssd_prep", ms, n * (C + 2 * H) * 8)
        prep(n, self.pos)
        seg, cnt = self.zero, self.i32([n])
        flops = 6.0 * n * H * d * dv       # two products with the state and the update
        for key, rows, count, pos, block in (("delta_prefill", n, cnt, self.pos, 8), ("delta_prefill_one_at_a_time", n, cnt, self.pos, 1),
                                             ("delta_decode", 1, self.one, self.last, 1)):
            ms = self.call("delta_recurrence", qk, v, gb, H, G, dp, dv, state, self.slot, pos, seg, count, 1, block, proj, ld, C, taps, mem, out)
            if rows > 1:
                self.res[key] = {"ms": round(ms, 4), "fp32_tflops": round(flops / ms / 1e9, 2), "frac_fp32_fma_nominal": round(flops / ms / 1e9 / FP32_TFLOPS, 4)}
            else:
                self.bytes_row(key, ms, 2 * H * dp * dv * 4)
        # the like kernels at the same heads and head sizes: a decay per key channel; a decay per head and token
        f, c, s0, sn = [self.i32(t) for t in scan_tiles(np.array([0]), np.array([n]), REC_TILE)]
        r_, k_, z_, w0, u = self.f32(n, H * d), self.f32(n, H * d), self.f32(n, H * d), self.bf(H * d), self.bf(H * d)
        hs, sh = self.f32(n, self.W), self.f32(1, self.W)
        cws = torch.zeros(int(L.ao_lm_channel_recurrence_workspace_bytes(len(f), n, H, d, dv)) // 4, device=self.dev)
        flops = 4.0 * n * H * d * dv
        for key, rows, tile, pos in (("fedipel_channel_recurrence_prefill", n, (f, c, len(f), s0, sn, 1, n, cws), self.pos),
                                     ("fedipel_channel_recurrence_decode", 1, (seg, self.one, 1, None, None, 0, 1, None), self.last)):
            ms = self.call("channel_recurrence", r_, H * d, k_, H * d, v, H * dv, z_, H * d, w0, u, BF16, H, d, dv, state, self.slot, pos, *tile, hs, sh, self.W, out,
                           H * dv)
            if rows > 1:
                self.res[key] = {"ms": round(ms, 4), "fp32_tflops": round(flops / ms / 1e9, 2), "frac_fp32_fma_nominal": round(flops / ms / 1e9 / FP32_TFLOPS, 4)}
            else:
                self.bytes_row(key, ms, 2 * H * d * dv * 4)
        ows = torch.zeros(int(L.ao_lm_outer_recurrence_workspace_bytes(len(f), n, H, d, dv)) // 4, device=self.dev)
        ms = self.call("outer_recurrence", r_, H * d, k_, H * d, v, H * dv, 0, sa, sb, H, None, None, H, H, d, dv, state, self.slot, self.pos, f, c, len(f), s0, sn, 1, n,
                       ows, out, H * dv)
        self.res["rutusun_outer_recurrence_prefill"] = {"ms": round(ms, 4), "fp32_tflops": round(flops / ms / 1e9, 2),
                                                        "frac_fp32_fma_nominal": round(flops / ms / 1e9 / FP32_TFLOPS, 4)}

    # ------------------------------------------------------------------------------------------------ row kernels
    def rows(self):
        n, W, ff, L = self.n, self.W, self.ff, self.L
        x, y, h, w = self.f32(n, W), self.f32(n, W) * 1e-3, self.bf(n, W), self.bf(W)
        ms = self.call("add_rms_norm", x, y, None, n, W, w, BF16, 1e-6, h)
        self.bytes_row("add_rms_norm", ms, n * W * 14)
        ms = self.call("add_layer_norm", x, y, 0.01, None, n, W, w, w, BF16, 1e-6, None, h)
        self.bytes_row("fedipel_add_layer_norm", ms, n * W * 14)
        up, ya = self.f32(n, ff), self.bf(n, ff)
        ms = self.call("xielu_rows", up, ff, n, ff, 0.7, 1.1, ya, ff, BF16)
        self.bytes_row("xielu_rows", ms, n * ff * 6)
        ms = self.call("unary_rows", up, F32, n, ff, 0, 0.0, None, 0, ya, BF16)
        self.bytes_row("fedipel_squared_relu_rows", ms, n * ff * 6)
        H, dv = self.delta.heads, self.delta.vdim
        rec, gate, go, nw = self.f32(n, H * dv), self.f32(n, H * dv), self.bf(n, H * dv + ff), self.bf(dv)
        ms = self.call("gated_group_norm_rows", rec, H * dv, gate, H * dv, 2, n, H * dv, H, nw, 1, BF16, 1e-6, go, H * dv + ff)
        self.bytes_row("gated_group_norm_rows", ms, n * H * dv * 10)


def kernel_numbers(name, prompt_len, decode_ctx):
    b = Bench(name, prompt_len, decode_ctx)
    b.latent()
    b.attention()
    b.recurrence()
    b.rows()
    return b.res


def run(sizes=(("Rigalorn-2k", "Fedipel-2k"), ("Rigalorn-4k", "Fedipel-4k")), prompt_len=2048, decode_ctx=1536, decode_steps=64):
    out = {"metric": "rigalorn_layers_prefill_decode", "dtype": "bf16", "data": "synthetic", "n_gpus": 1, "sizes": {}}
    for names in sizes:
        out["sizes"][names[0]] = {"models": model_numbers(names, prompt_len, decode_ctx, decode_steps),
                                  "kernels": kernel_numbers(names[0], prompt_len, decode_ctx)}
        torch.cuda.empty_cache()
    return out


if __name__ == "__main__":
    print(json.dumps(run()))
