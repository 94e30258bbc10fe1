"""Prefill and decode throughput of Sozanex layers at sizes of real models (random weights), beside the framework's closest
existing family — Rigalorn, with the two of its mixers that are softmax attention — at equal size in bf16, and the design's own
kernels timed alone against their roofline, each beside the like kernel of an existing family.
`python bench.py --workload sozanex-layers` prints the result as one JSON line; this file is the measurement.

Timing as in rigalorn_bench.py: CUDA events after 3 warm-up runs; model inputs and weights exceed L2, the kernel-alone timings
write a 256 MB buffer between runs.
"""
import ctypes
import json
import os
import sys

import numpy as np
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

from benchmarks.bitipel_bench import timed  # noqa: E402
from benchmarks.rigalorn_bench import BF16, F32, Bench, model_numbers  # noqa: E402


def rigalorn_of_two(name):
    """The named Rigalorn configuration with its latent attention and attention layers only."""
    from torchao_fork_b200._models.rigalorn import Rigalorn, rigalorn_configs
    cfg = rigalorn_configs[name]()
    cfg.layers = [la for la in cfg.layers if la.type != "delta"]
    for la in cfg.layers:       # nothing to mix a single attention layer's values with
        if la.type == "attention":
            la.mixer.v_mix = False
    return Rigalorn.random_init(cfg, torch.device("cuda"), torch.bfloat16)


class SozanexBench(Bench):
    def __init__(self, name, prompt_len, decode_ctx):
        from torchao_fork_b200._models.sozanex import sozanex_configs
        self.setup(sozanex_configs[name](), prompt_len, decode_ctx)
        del self.res["fp32_fma_tflops_nominal"]

    # ------------------------------------------------------------------------------------------------ latent attention
    def latent(self):
        a, n, L = self.lat, self.n, self.L
        H, dn, dr, dv, R, Rq = a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank
        qn, qr, kr, out = self.bf(H, n, dn), self.f32(n, H, dr), self.bf(n, dr), self.bf(n, H * dv)
        ld, ldp = H * (dn + dv), H * dv + Rq + R + dr
        kv, sink, proj = self.bf(n, ld), self.bf(H), self.f32(n, ldp)
        rows = ctypes.c_int()
        L.ao_lm_latent_attention_expanded_plan(BF16, dn, dr, dv, ctypes.byref(rows))
        tf, tc, nt = self.tiles(rows.value)
        key0 = self.i32(np.zeros(nt))
        pairs = n * (n + 1) / 2
        flops, issued = 2.0 * pairs * H * (dn + dr + dv), 2.0 * pairs * H * (dn + 2 * dr + 3 * dv)
        head = (qn, qr, kv, ld, kv.data_ptr() + 2 * H * dn, ld, kr, BF16, self.pos, tf, tc, key0, nt, n, H, dn, dr, dv, a.scale, n)
        self.tensor_row("latent_prompt_sink_and_gate", self.call("gated_latent_attention_expanded", *head, sink, proj, ldp, out, H * dv), flops, issued)
        self.tensor_row("rigalorn_latent_prompt", self.call("window_latent_attention_expanded", *head, None, None, out, H * dv), flops, issued)
        # one decoded token over the cached latents, key splits as the step function picks them
        S, ctx = self.ctx + 64, self.ctx
        ring_c, ring_kr, c1, kr1 = self.bf(1, S, R), self.bf(1, S, dr), self.bf(1, R), self.bf(1, dr)
        qa, qr1, olat = self.f32(H, 1, R), self.f32(1, H, dr), self.bf(1, H, R)
        ns = max(1, min(-(-S // 32), -(-4 * 148 // -(-H // 16)), 64))
        ws = torch.zeros(int(L.ao_lm_latent_attention_workspace_bytes(1, H, R, ns)), dtype=torch.uint8, device=self.dev)
        for key, sk in (("latent_decode_sink", sink), ("rigalorn_latent_decode", None)):
            ms = self.call("window_latent_attention", qa, qr1, ring_c, ring_kr, c1, kr1, BF16, S, self.zero, self.last, self.zero, self.zero, self.one, 1,
                           1, H, R, dr, a.scale, S, sk, None, ns, ws, ws.numel(), olat)
            self.bytes_row(key, ms, ctx * (R + dr) * 2, splits=ns)
        uv = self.bf(H, dv, R)
        row = self.bf(1, H * dv)
        ms = self.call("latent_value_up", olat, uv, BF16, 1, H, R, dv, proj, ldp, row, H * dv)
        self.bytes_row("latent_value_up_with_gate_decode", ms, uv.numel() * 2)
        heads = row.as_strided((H, 1, dv), (dv, H * dv, 1))
        ms = timed(lambda: torch.bmm(olat.transpose(0, 1), uv.transpose(1, 2), out=heads), flush=self.flush)
        self.bytes_row("batched_product_without_gate_decode", ms, uv.numel() * 2)
        q1, qr0 = self.f32(1, H, dn + dr), self.f32(1, H, dr)
        uk = self.bf(H, dn, R)
        ms = self.call("latent_query_fold", q1, uk, BF16, 1, H, dn, dr, R, a.rot.dims, a.rot.inv_freq(self.dev), 1.1, self.last, qa, qr0)
        self.bytes_row("latent_query_fold_decode", ms, uk.numel() * 2)
        # row kernels around it
        wq, wc, inv = self.bf(Rq), self.bf(R), a.rot.inv_freq(self.dev)
        cq, c, krr, cc, ck = self.bf(n, Rq), self.bf(n, R), self.bf(n, dr), self.bf(1, n, R), self.bf(1, n, dr)
        ms = self.call("latent_low_prep_store", proj, ldp, n, H * dv, Rq, H * dv + Rq, R, dr, wq, wc, BF16, 1e-6, a.rot.dims, inv, 1.1, self.pos, self.slot,
                       n, cq, c, krr, cc, ck)
        self.bytes_row("latent_low_prep_store", ms, n * (Rq * 6 + (R + dr) * 8))
        q = self.f32(n, H * (dn + dr))
        ms = self.call("latent_query_prep", q, n, H, dn, dr, BF16, a.rot.dims, inv, 1.1, self.pos, qn, qr)
        self.bytes_row("latent_query_prep", ms, n * H * (dn * 6 + dr * 8))

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
        self.tensor_row("window_prompt_as_in_rigalorn", ms, 2.0 * pairs * H * (d + dv), 2.0 * pairs * H * (d + 3 * dv))
        ns = max(1, min(-(-C // 32), -(-4 * 148 // G), 64))
        ws = torch.zeros(max(16, int(L.ao_lm_window_attention_workspace_bytes(1, 1, H, G, dv, ns))), dtype=torch.uint8, device=self.dev)
        ms = self.call("window_attention", qn, kn, vn, rk, rv, None, None, C, 0, BF16, self.zero, self.last, self.zero, self.zero, self.one, 1, 1, H, G, d, dv,
                       C, 0, a.scale, 0.0, 0, 0.0, 1.0, ns, ws, ws.numel(), out, H * dv)
        self.bytes_row("window_decode_as_in_rigalorn", ms, self.ctx * G * (d + dv) * 2, splits=ns)
        ldq = (H + G) * d + G * dv
        pr, inv = self.f32(n, ldq), a.rot.inv_freq(self.dev)
        qb, kb, vb, w = self.bf(H * d), self.bf(G * d), self.bf(G * dv), self.bf(d)
        byts = n * (ldq * 4 + H * d * 4 + G * (d + dv) * 2)
        ms = self.call("qkv_norm_rotary_prep", pr, ldq, 0, H * d, (H + G) * d, qb, kb, vb, w, w, 1e-6, self.pos, inv, a.rot.dims, 1, 1.0, n, H, G, d, G * dv,
                       BF16, qn, kn, vn, None, 0, None, None)
        self.bytes_row("qkv_norm_rotary_prep", ms, byts)
        ms = self.call("qkv_rotary_mix_prep", pr, ldq, 0, H * d, (H + G) * d, qb, kb, vb, self.pos, inv, a.rot.dims, 1, 1.0, None, 0.0, n, H, G, d, G * dv, BF16,
                       qn, kn, vn)
        self.bytes_row("rigalorn_qkv_rotary_mix_prep", ms, byts)
        ms = self.call("qk_norm_prep", pr, ldq, 0, H * d, (H + G) * d, qb, kb, vb, w, w, 0.0, 1, self.pos, self.slot, None, None, 0, n, H, G, d, dv, 1e-6, BF16,
                       qn, kn, vn)
        self.bytes_row("rutusun_qk_norm_prep", ms, byts)

    # ------------------------------------------------------------------------------------------------ row kernels
    def rows(self):
        n, W, ff = self.n, self.W, self.ff
        x, y, h, w, yb = self.f32(n, W), self.f32(n, W) * 1e-3, self.bf(n, W), self.bf(W), self.f32(W)
        ms = self.call("post_layer_norm_residual", x, y, W, yb, w, None, 0, 0, w, BF16, 1e-6, n, W, h, W)
        self.bytes_row("post_layer_norm_residual", ms, n * W * 14)
        ms = self.call("post_layer_norm_residual", x, y, W, None, None, y, W, 1, w, BF16, 1e-6, n, W, h, W)
        self.bytes_row("post_layer_norm_residual_pass_input", ms, n * W * 14)
        ms = self.call("postnorm_residual", x, y, F32, yb, w, None, None, w, BF16, 1e-6, n, W, h)
        self.bytes_row("rutusun_postnorm_residual", ms, n * W * 14)
        ms = self.call("add_rms_norm", x, y, None, n, W, w, BF16, 1e-6, h)
        self.bytes_row("rigalorn_add_rms_norm", ms, n * W * 14)
        ms = self.call("add_layer_norm", x, None, 0.0, None, n, W, w, None, BF16, 1e-6, None, h)
        self.bytes_row("final_layer_norm", ms, n * W * 6)
        ms = self.call("add_rms_norm", x, None, None, n, W, w, BF16, 1e-6, h)
        self.bytes_row("rigalorn_final_rms_norm", ms, n * W * 6)
        b = self.cfg.bigram
        table, big = self.bf(self.cfg.vocab_size, W), self.bf(b.buckets + 1, W)
        tok = torch.randint(0, self.cfg.vocab_size, (n,), device=self.dev)
        last = torch.zeros(1, dtype=torch.int64, device=self.dev)
        ahead = self.i32(np.arange(n - 1, -1, -1))
        ms = self.call("embed_bigram", table, big, BF16, tok, n, W, 1.0, b.buckets, b.mul_prev, b.mul_cur, last, self.slot, self.pos, self.back, ahead, x, h)
        self.bytes_row("embed_bigram", ms, n * W * 10)
        ms = self.call("embed_scaled", table, BF16, tok, n, W, 1.0, x)
        self.bytes_row("rigalorn_embed_scaled", ms, n * W * 6)
        up, ya, f = self.bf(n, ff), self.bf(n, ff), self.f32(n, ff)
        ms = self.call("unary_rows", up, BF16, n, ff, 0, 0.0, None, 0, ya, BF16)
        self.bytes_row("squared_relu_rows", ms, n * ff * 4)
        ms = self.call("xielu_rows", f, ff, n, ff, 0.7, 1.1, ya, ff, BF16)
        self.bytes_row("rigalorn_xielu_rows", ms, n * ff * 6)

    # ------------------------------------------------------------------------------------------------ products of one row
    def products(self):
        W, ff = self.W, self.ff
        for key, M, K, act in (("up", ff, W, 1), ("down", W, ff, 0), ("o", W, W, 0), ("head", self.cfg.vocab_size, W, 0)):
            x, w = self.bf(1, K), self.bf(M, K)
            out = self.bf(1, M) if act else self.f32(1, M)
            ms = self.call("gemv_rows", x, K, w, K, 1, M, K, act, out, M)
            self.bytes_row(f"gemv_rows_{key}_one_row", ms, M * K * 2)
            ms = timed(lambda: torch.mm(x, w.t(), out_dtype=torch.float32), flush=self.flush)
            self.bytes_row(f"library_product_{key}_one_row", ms, M * K * 2)


def kernel_numbers(name, prompt_len, decode_ctx):
    b = SozanexBench(name, prompt_len, decode_ctx)
    b.latent()
    b.attention()
    b.rows()
    b.products()
    return b.res


def run(sizes=("2k", "4k"), prompt_len=2048, decode_ctx=1536, decode_steps=64):
    out = {"metric": "sozanex_layers_prefill_decode", "dtype": "bf16", "data": "synthetic", "n_gpus": 1, "sizes": {}}
    for s in sizes:
        names = [f"Sozanex-{s}", f"Rigalorn-{s} (latent attention, attention)"] + (["Sozanex-2k-loop"] if s == "2k" else [])
        out["sizes"][names[0]] = {"models": model_numbers(names, prompt_len, decode_ctx, decode_steps, {names[1]: lambda s=s: rigalorn_of_two(f"Rigalorn-{s}")}),
                                  "kernels": kernel_numbers(names[0], prompt_len, decode_ctx)}
        torch.cuda.empty_cache()
    return out


if __name__ == "__main__":
    print(json.dumps(run()))
