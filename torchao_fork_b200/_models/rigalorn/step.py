"""The step function of Rigalorn: runs the tokens a step brings — any mix of prompt portions and single decoded tokens of
several sequences — through the model's layers on the state that earlier steps left, as launches of libao_b200_lm
kernels (include/ao_b200_lm.h) and library GEMMs for the dense projections.

The residual x is fp32.  Mixer and feed-forward of a layer read the same norm output and add into the same residual, so a
layer is
    ONE GEMM for every projection of the row, the feed-forward's up-projection included (fp32 result)
    -> the mixer's kernels, which leave their heads in the first columns of a row [heads | units]
    -> `xielu_rows`, which leaves the feed-forward's units in the other columns
    -> ONE GEMM with [W_o | W_down] (its sum over the row IS mixer + feed-forward, fp32 result)
    -> `add_rms_norm`: x += result, and the next layer's norm while the row is on chip.
The mixers between the two GEMMs:
  attention: `qkv_rotary_mix_prep` (biases, scaled rotation, the first value-mixing layer's values mixed in) ->
      `window_attention` / `window_attention_prompt` over the ring and the step's own rows -> `window_append`.
  delta: `delta_prep` (convolutions, SiLU, unit vectors, decays, step sizes) -> `delta_recurrence` (matrix state per slot; also
      saves the convolutions' last inputs) -> `gated_group_norm_rows` (unit RMS per head, weight, SiLU gate).
  latent_attention: `latent_low_prep` (both latent norms, rotated shared key part) -> GEMM W_uq -> `latent_query_prep` -> then
      for prompt portions: the visible latents made contiguous, ONE GEMM for all heads' keys and values,
          `window_latent_attention_expanded`;
      for few rows: batched GEMM that folds the key up-projection into the queries, `window_latent_attention` over the latents
          themselves, batched GEMM with the value up-projection;
      -> `ring_append`.
Norms, rotations, attention scores and weights, decays, step sizes, unit vectors and recurrent states are fp32 in both
storage types.

`StepEngine.step` is what prefill, the trace runner and tests call; `GraphDecodeEngine` wraps the same layer loop for
one token per sequence with all metadata in device memory, captured into a CUDA graph.
"""
import ctypes

import numpy as np
import torch

from ... import _lib
from ..segment_step import GraphDecodeEngine, SegmentStepEngine, StepMeta, _p  # noqa: F401
from .model import UNIT_EPS, Rigalorn

PAIR_HALVES = 1                           # rotation couples (i, i + dims / 2)
GATE_SILU_AFTER_NORM = 2                  # mode of gated_group_norm
# prompt portions attend over expanded keys and values of at most this many bytes per layer; beyond it in the folded form
EXPAND_MAX_BYTES = 4 << 30


class StepEngine(SegmentStepEngine):
    def __init__(self, model: Rigalorn):
        super().__init__(model)
        self.windows = sorted({s[-1] for s in self.attn_keys if s[0] == "latent"})

    # ------------------------------------------------------------------------------------------------ plans
    def _shape(self, la, ls):
        a = la.mixer
        if la.type == "attention":
            return ("window", a.heads, a.kv_heads, a.dim, a.vdim)
        return ("latent", a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, min(a.window, ls.latent.c.shape[1]))

    def _attention_shapes(self):
        return sorted({self._shape(la, ls) for la, ls in zip(self.cfg.layers, self.m.run_state) if la.type != "delta"})

    def _attention_plan(self, shape):
        rows, prompt = ctypes.c_int(), ctypes.c_int()
        if shape[0] == "window":
            _, H, G, d, dv = shape
            _lib.lm_check(self.L.ao_lm_window_attention_plan(self.dt, 1, H, G, d, dv, ctypes.byref(rows)), "window_attention_plan")
            _lib.lm_check(self.L.ao_lm_window_attention_prompt_plan(self.dt, 1, H, G, d, dv, ctypes.byref(prompt)), "window_attention_prompt_plan")
        else:
            _, H, dn, dr, dv, R, _ = shape
            _lib.lm_check(self.L.ao_lm_latent_attention_plan(self.dt, H, R, dr, ctypes.byref(rows)), "latent_attention_plan")
            _lib.lm_check(self.L.ao_lm_latent_attention_expanded_plan(self.dt, dn, dr, dv, ctypes.byref(prompt)), "latent_attention_expanded_plan")
        return rows.value, 1 << 30, prompt.value      # tiles may cross any position

    @staticmethod
    def _history(pos0, window):
        """Keys from earlier steps that a segment starting at position pos0 can see."""
        return np.minimum(pos0, window - 1)

    def _prompt_form(self, shape, starts, counts, pos):
        if shape[0] != "latent":
            return True
        _, H, dn, _, dv, _, window = shape
        return int((self._history(pos[starts], window) + counts).sum()) * H * (dn + dv) * 2 <= EXPAND_MAX_BYTES

    def _piece_tables(self, starts, counts, slot, pos, forms, tiles):
        """For every window of latent-attention layers that attend in the expanded form: ("rows", window) = where each
        contiguous latent row comes from (absent when the step's own rows are all of them), ("key0", window) = per tile, the
        row that key 0 of its sequence would have."""
        out = {}
        for shape, form in forms.items():
            if shape[0] != "latent" or not form[2] or ("key0", shape[-1]) in out:
                continue
            window = shape[-1]
            hist = self._history(pos[starts], window)
            base = np.concatenate([[0], np.cumsum(hist + counts)[:-1]])            # a segment's first contiguous row
            first = tiles[form][0]
            seg = np.searchsorted(starts, first, side="right") - 1
            out[("key0", window)] = (base - (pos[starts] - hist))[seg].astype(np.int32)
            if hist.any():
                parts = []
                for s, c, h in zip(starts, counts, hist):
                    p0 = int(pos[s])
                    parts += [-1 - (int(slot[s]) * window + np.arange(p0 - h, p0) % window), np.arange(s, s + c)]
                out[("rows", window)] = np.concatenate(parts).astype(np.int32)
        return out

    # ------------------------------------------------------------------------------------------------ layers
    def _norm(self, x, y, w, st):
        """x += y (None: nothing added); -> RMS norm of x with weight w in the model's dtype (w None: only the add)."""
        n, W = x.shape
        h = None if w is None else torch.empty(n, W, dtype=self.m.dtype, device=self.dev)
        _lib.lm_check(self.L.ao_lm_add_rms_norm(_p(x), _p(y), None, n, W, _p(w), self.dt, self.cfg.norm_eps, _p(h), st), "add_rms_norm")
        return h

    def _layers(self, d_tok: torch.Tensor, meta: StepMeta, after_run=None) -> torch.Tensor:
        m, cfg, L, dt, dev = self.m, self.cfg, self.L, self.dt, self.dev
        n, W = meta.n, cfg.width
        st = torch.cuda.current_stream(dev).cuda_stream
        x = torch.empty(n, W, dtype=torch.float32, device=dev)
        _lib.lm_check(L.ao_lm_embed_scaled(_p(m.embed), dt, _p(d_tok), n, W, cfg.embedding_scale, _p(x), st), "embed_scaled")
        layers = m.layers
        if not layers:
            self.launches = 1
            return x
        h = self._norm(x, None, layers[0].norm1, st)
        launches = 2
        v_first = None                  # the step's values of the first value-mixing layer
        for i, lay in enumerate(layers):
            la, ls = lay.args, m.run_state[i]
            proj = self._mm_f32(h, lay.w_in)
            row = torch.empty(n, lay.w_out.shape[1], dtype=m.dtype, device=dev)       # [heads | units]
            if la.type == "attention":
                mixed, c = self._attention(lay, la, ls, proj, row, v_first if la.mixer.v_mix else None, meta, st)
                if la.mixer.v_mix and v_first is None:
                    v_first = mixed
            elif la.type == "delta":
                c = self._delta(lay, la.mixer, ls, proj, row, meta, st)
            else:
                c = self._latent(lay, la, ls, proj, row, meta, st)
            if la.ff:
                esz = row.element_size()
                _lib.lm_check(L.ao_lm_xielu_rows(proj.data_ptr() + 4 * lay.up_off, lay.ld, n, la.ff, lay.act_pos, lay.act_neg,
                                                 row.data_ptr() + esz * lay.o_width, row.shape[1], dt, st), "xielu_rows")
                c += 1
            y = self._mm_f32(row, lay.w_out)
            nw = layers[i + 1].norm1 if i + 1 < len(layers) else None
            if after_run is not None:       # the residual as the layer leaves it
                self._norm(x, y, None, st)
                after_run(i, x)
                h = self._norm(x, None, nw, st) if nw is not None else None
                c += 1
            else:
                h = self._norm(x, y, nw, st)
            launches += c + 3
        self.launches = launches
        return x

    def _attention(self, lay, la, ls, proj, row, v_first, meta: StepMeta, st):
        """Softmax attention under a window into the first columns of `row` -> (the step's values as cached, launches)."""
        L, dt, dev, tdt, a = self.L, self.dt, self.dev, self.m.dtype, la.mixer
        H, G, d, dv, n, cache = a.heads, a.kv_heads, a.dim, a.vdim, meta.n, ls.window
        qn = torch.empty(n, H, d, dtype=torch.float32, device=dev)
        kn, vn = torch.empty(n, G, d, dtype=tdt, device=dev), torch.empty(n, G, dv, dtype=tdt, device=dev)
        _lib.lm_check(L.ao_lm_qkv_rotary_mix_prep(_p(proj), lay.ld, lay.q_off, lay.k_off, lay.v_off, _p(lay.q_b), _p(lay.k_b), _p(lay.v_b),
                                                  _p(meta.pos), _p(lay.inv_freq), a.rot.dims, PAIR_HALVES, a.rot.amplitude, _p(v_first),
                                                  lay.lam, n, H, G, d, G * dv, dt, _p(qn), _p(kn), _p(vn), st), "qkv_rotary_mix_prep")
        tf, tc, nt, tensor = meta.attn[self._shape(la, ls)]
        window = min(a.window, cache.ring)
        common = (_p(qn), _p(kn), _p(vn), _p(cache.k), _p(cache.v), _p(cache.k_first), _p(cache.v_first), cache.ring, 0, dt, _p(meta.slot),
                  _p(meta.pos), _p(meta.back), _p(tf), _p(tc), nt, 1, H, G, d, dv, window, 0, a.scale, 0.0, 0, 0.0, 1.0)
        c = 3
        if tensor:      # prompt portions: the tensor-core form
            _lib.lm_check(L.ao_lm_window_attention_prompt(*common, _p(row), row.shape[1], st), "window_attention_prompt")
        else:
            ns = self._splits(nt * G, window)    # few rows over a long window: the keys are shared out over more CTAs
            ws = torch.empty(max(16, int(L.ao_lm_window_attention_workspace_bytes(nt, 1, H, G, dv, ns))), dtype=torch.uint8, device=dev)
            _lib.lm_check(L.ao_lm_window_attention(*common, ns, _p(ws), ws.numel(), _p(row), row.shape[1], st), "window_attention")
            c += 1 if ns > 1 else 0
        _lib.lm_check(L.ao_lm_window_append(_p(kn), _p(vn), n, G * d, G * dv, cache.ring, 0, dt, _p(meta.slot), _p(meta.pos), _p(meta.ahead),
                                            _p(cache.k), _p(cache.v), _p(cache.k_first), _p(cache.v_first), st), "window_append")
        return vn, c

    def _delta(self, lay, a, ls, proj, row, meta: StepMeta, st):
        """Gated delta rule into the first columns of `row` -> launches."""
        L, dt, dev = self.L, self.dt, self.dev
        H, G, d, dp, dv, n = a.heads, a.kv_heads, a.dim, a.padded_dim, a.vdim, meta.n
        f32 = dict(dtype=torch.float32, device=dev)
        qk, v, gb = torch.empty(n, 2, G, dp, **f32), torch.empty(n, H * dv, **f32), torch.empty(n, H, 2, **f32)
        _lib.lm_check(L.ao_lm_delta_prep(_p(proj), lay.ld, 0, lay.a_off, lay.b_off, n, H, G, d, dp, dv, a.taps, _p(lay.conv_w),
                                         _p(ls.conv.x), _p(meta.slot), _p(meta.pos), _p(meta.back), _p(lay.a_log), _p(lay.dt_bias), dt,
                                         UNIT_EPS, d ** -0.5, _p(qk), _p(v), _p(gb), st), "delta_prep")
        rec = torch.empty(n, H * dv, **f32)
        sf, sc, ns = meta.seg
        _lib.lm_check(L.ao_lm_delta_recurrence(_p(qk), _p(v), _p(gb), H, G, dp, dv, _p(ls.mat.s), _p(meta.slot), _p(meta.pos), _p(sf), _p(sc),
                                               ns, 1 if ns == n else 8, _p(proj), lay.ld, a.channels, a.taps, _p(ls.conv.x), _p(rec), st),
                      "delta_recurrence")
        _lib.lm_check(L.ao_lm_gated_group_norm_rows(_p(rec), H * dv, proj.data_ptr() + 4 * lay.g_off, lay.ld, GATE_SILU_AFTER_NORM, n, H * dv,
                                                    H, _p(lay.mix_norm), 1, dt, self.cfg.norm_eps, _p(row), row.shape[1], st),
                      "gated_group_norm_rows")
        return 3

    def _latent(self, lay, la, ls, proj, row, meta: StepMeta, st):
        """Latent attention under a window into the first columns of `row` -> launches."""
        L, dt, dev, tdt, a, cache = self.L, self.dt, self.dev, self.m.dtype, la.mixer, ls.latent
        H, dn, dr, dv, R, Rq, n = a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank, meta.n
        act = dict(dtype=tdt, device=dev)
        cq, c, kr = torch.empty(n, Rq, **act), torch.empty(n, R, **act), torch.empty(n, dr, **act)
        rot = (a.rot.dims, _p(lay.inv_freq), a.rot.amplitude)
        _lib.lm_check(L.ao_lm_latent_low_prep(_p(proj), lay.ld, n, lay.q_off, Rq, lay.kv_off, R, dr, _p(lay.q_norm), _p(lay.c_norm), dt,
                                              self.cfg.norm_eps, *rot, _p(meta.pos), _p(cq), _p(c), _p(kr), st), "latent_low_prep")
        q = self._mm_f32(cq, lay.uq)
        qn, qr = torch.empty(H, n, dn, **act), torch.empty(n, H, dr, dtype=torch.float32, device=dev)
        _lib.lm_check(L.ao_lm_latent_query_prep(_p(q), n, H, dn, dr, dt, *rot, _p(meta.pos), _p(qn), _p(qr), st), "latent_query_prep")
        shape = self._shape(la, ls)
        ring, window = cache.c.shape[1], shape[-1]
        tf, tc, nt, tensor = meta.attn[shape]
        launches = 4
        if tensor:
            launches += self._latent_expanded(lay, a, cache, c, kr, qn, qr, row, tf, tc, nt, window, meta, st)
        else:
            qa = self._bmm_f32(qn, lay.uk)                                             # fp32 [H][n][R]
            ns = self._splits(nt * -(-H // 16), window)
            ws = torch.empty(max(16, int(L.ao_lm_latent_attention_workspace_bytes(n, H, R, ns))), dtype=torch.uint8, device=dev)
            olat = torch.empty(n, H, R, **act)
            _lib.lm_check(L.ao_lm_window_latent_attention(_p(qa), _p(qr), _p(cache.c), _p(cache.kr), _p(c), _p(kr), dt, ring, _p(meta.slot),
                                                          _p(meta.pos), _p(meta.back), _p(tf), _p(tc), nt, n, H, R, dr, a.scale, window,
                                                          None, None, ns, _p(ws), ws.numel(), _p(olat), st), "window_latent_attention")
            heads = row.as_strided((H, n, dv), (dv, row.shape[1], 1))
            torch.bmm(olat.transpose(0, 1), lay.uv.transpose(1, 2), out=heads)
            launches += 4 if ns > 1 else 3
        _lib.lm_check(L.ao_lm_ring_append(_p(c), _p(kr), n, R, dr, ring, dt, _p(meta.slot), _p(meta.pos), _p(meta.ahead), _p(cache.c),
                                          _p(cache.kr), st), "ring_append")
        return launches

    def _latent_expanded(self, lay, a, cache, c, kr, qn, qr, row, tf, tc, nt, window, meta, st):
        """Prompt portions: every sequence's visible latents up-projected into per-head keys and values -> launches."""
        L, dt, dev, tdt = self.L, self.dt, self.dev, self.m.dtype
        H, dn, dr, dv, R, n = a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, meta.n
        src, launches = meta.extra.get(("rows", window)), 2
        if src is not None:
            ca, kra = torch.empty(len(src), R, dtype=tdt, device=dev), torch.empty(len(src), dr, dtype=tdt, device=dev)
            _lib.lm_check(L.ao_lm_latent_rows_gather(_p(src), len(src), _p(c), _p(kr), _p(cache.c), _p(cache.kr), dt, R, dr, _p(ca),
                                                     _p(kra), st), "latent_rows_gather")
            c, kr, launches = ca, kra, 3
        kv = torch.mm(c, lay.ukv.t())                                                  # [rows][H dn | H dv]
        ld = H * (dn + dv)
        _lib.lm_check(L.ao_lm_window_latent_attention_expanded(
            _p(qn), _p(qr), _p(kv), ld, kv.data_ptr() + kv.element_size() * H * dn, ld, _p(kr), dt, _p(meta.pos), _p(tf), _p(tc),
            _p(meta.extra[("key0", window)]), nt, n, H, dn, dr, dv, a.scale, window, None, None, _p(row), row.shape[1], st),
            "window_latent_attention_expanded")
        return launches

    def _bmm_f32(self, a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """[b][n][K] x [b][K][M] -> fp32 [b][n][M]."""
        return torch.bmm(a, w, out_dtype=torch.float32) if a.dtype == torch.bfloat16 else torch.bmm(a, w)

    def _logits_dev(self, x, d_rows, k, out=None):
        m, cfg = self.m, self.cfg
        st = torch.cuda.current_stream(self.dev).cuda_stream
        xn = torch.empty(k, cfg.width, dtype=m.dtype, device=self.dev)
        _lib.lm_check(self.L.ao_lm_add_rms_norm(_p(x), None, _p(d_rows), k, cfg.width, _p(m.final_norm), self.dt, cfg.norm_eps, _p(xn), st),
                      "add_rms_norm")
        lg = self._mm_f32(xn, m.head)
        if out is not None:
            out.copy_(lg)
            return out
        return lg
