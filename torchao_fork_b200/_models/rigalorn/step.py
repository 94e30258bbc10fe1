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
import torch

from ... import _lib
from ..segment_step import GraphDecodeEngine, StepMeta, _p  # noqa: F401
from ..softmax_step import PAIR_HALVES, SoftmaxStepEngine
from .model import UNIT_EPS, Rigalorn

GATE_SILU_AFTER_NORM = 2                  # mode of gated_group_norm


class StepEngine(SoftmaxStepEngine):
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
        c = 2 + self._window_attend(a, self._shape(la, ls), cache, qn, kn, vn, row, meta, st)
        self._window_append(a, cache, kn, vn, meta, st)
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
        shape = self._shape(la, ls)
        q, qr, k = self._latent_queries(lay, a, shape, cq, meta, st)
        launches = 2 + k + self._latent_attend(lay, a, shape, cache, c, kr, q, qr, row, meta, st)
        _lib.lm_check(L.ao_lm_ring_append(_p(c), _p(kr), n, R, dr, cache.c.shape[1], dt, _p(meta.slot), _p(meta.pos), _p(meta.ahead),
                                          _p(cache.c), _p(cache.kr), st), "ring_append")
        return launches

    def _logits_dev(self, x, d_rows, k, out=None):
        m, cfg = self.m, self.cfg
        st = torch.cuda.current_stream(self.dev).cuda_stream
        xn = torch.empty(k, cfg.width, dtype=m.dtype, device=self.dev)
        _lib.lm_check(self.L.ao_lm_add_rms_norm(_p(x), None, _p(d_rows), k, cfg.width, _p(m.final_norm), self.dt, cfg.norm_eps, _p(xn), st),
                      "add_rms_norm")
        return self._mm_f32(xn, m.head, out)
