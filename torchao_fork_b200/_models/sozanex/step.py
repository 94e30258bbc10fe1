"""The step function of Sozanex: runs the tokens a step brings — any mix of prompt portions and single decoded tokens of
several sequences — through the model's layer runs on the state that earlier steps left, as launches of libao_b200_lm
kernels (include/ao_b200_lm.h) and library GEMMs for the dense projections.

The residual x is fp32.  Every sublayer ends in ONE row kernel (`post_layer_norm_residual`): the sublayer's result (with its
projection's bias) enters x through its own layer norm, and the next sublayer's input norm is taken while the row is in
registers.
  embedding: `embed_bigram` (scaled row + hashed row of the token pair; keeps the slot's last token).
  a pass over the looped span: W_in [x; x0] as W_a x + W_b x0.  W_b x0 is made once per step; the row kernel that closes the
      layer in front of a pass leaves x in the storage type, ONE GEMM makes W_a x, and the row kernel adds the two into the new
      residual with the pass's first norm.
  attention: ONE GEMM [q | k | v] (fp32 result) -> `qkv_norm_rotary_prep` (biases, RMS norm per head, scaled rotation; for
      single decoded tokens also the ring's new rows) -> `window_attention` / `window_attention_prompt` over the ring and the
      step's own rows -> `window_append` (prompt portions) -> GEMM W_o.
  latent_attention: ONE GEMM [gate | dq | dkv] (fp32 result) -> `latent_low_prep_store` (both latent norms, rotated shared key
      part, the cache's new rows) -> GEMM W_uq -> `latent_query_prep` -> then
      for prompt portions: the visible latents made contiguous, ONE GEMM for all heads' keys and values,
          `gated_latent_attention_expanded` (sink in the denominator, sigmoid gate on the way out);
      for few rows: `latent_query_fold` instead (the key up-projection folded into the queries), `window_latent_attention` over the
          latents themselves (sink), `latent_value_up` (value up-projection and sigmoid gate);
      -> GEMM W_o.
  feed-forward: GEMM up -> squared ReLU -> GEMM down.
For up to eight rows in bf16 every product is `gemv_rows`, whose weights travel while the kernel in front finishes; the one in front
of the squared ReLU has it built in.
Norms, rotations, attention scores and weights, and the residual are fp32 in both storage types.

`StepEngine.step` is what prefill, the trace runner and tests call; `GraphDecodeEngine` wraps the same layer loop for
one token per sequence with all metadata in device memory, captured into a CUDA graph.
"""
import torch

from ... import _lib
from ..experts import act_unit
from ..segment_step import GraphDecodeEngine, StepMeta, _p  # noqa: F401
from ..softmax_step import PAIR_HALVES, SoftmaxStepEngine
from .model import Sozanex


class StepEngine(SoftmaxStepEngine):
    def __init__(self, model: Sozanex):
        super().__init__(model)
        self._normed = None     # a decode step's rows behind the output norm
        self.plan = [(r, i, begins) for r, (i, begins) in enumerate(self.cfg.schedule)]

    def _layer_runs(self):
        return [(self.cfg.layers[i], rs) for i, rs in zip(self.cfg.runs, self.m.run_state)]

    # ------------------------------------------------------------------------------------------------ layers
    def _close(self, x, y, post_w, y_bias, next_w, st, cast=False, add=None):
        """x += norm(y + y_bias) * post_w (y None: x stays; add given: x = y + add) -> norm(x) * next_w in the model's dtype, x
        itself in that dtype (cast), or nothing.  y, add: fp32 [n][W], rows of any stride."""
        n, W = x.shape
        out = torch.empty(n, W, dtype=self.m.dtype, device=self.dev) if next_w is not None or cast else None
        _lib.lm_check(self.L.ao_lm_post_layer_norm_residual(
            _p(x), _p(y), y.stride(0) if y is not None else 0, _p(y_bias), _p(post_w), _p(add), add.stride(0) if add is not None else 0,
            0 if add is None else 1, _p(next_w), self.dt, self.cfg.norm_eps, n, W, _p(out), W, st), "post_layer_norm_residual")
        return out

    def _layers(self, d_tok: torch.Tensor, meta: StepMeta, after_run=None) -> torch.Tensor:
        m, cfg, L, dt, dev = self.m, self.cfg, self.L, self.dt, self.dev
        n, W = meta.n, cfg.width
        st = torch.cuda.current_stream(dev).cuda_stream
        x = torch.empty(n, W, dtype=torch.float32, device=dev)
        x0 = torch.empty(n, W, dtype=m.dtype, device=dev) if cfg.loop else None      # the embedding output as a product's operand
        b = cfg.bigram
        _lib.lm_check(L.ao_lm_embed_bigram(_p(m.embed), _p(m.bigram), dt, _p(d_tok), n, W, cfg.embedding_scale, b.buckets if b else 0,
                                           b.mul_prev if b else 0, b.mul_cur if b else 0, _p(m.run_state[-1].last.token) if b else None,
                                           _p(meta.slot), _p(meta.pos), _p(meta.back), _p(meta.ahead), _p(x), _p(x0), st), "embed_bigram")
        launches = 1
        if not self.plan:
            self.launches = launches
            return x
        y0 = None
        if cfg.loop:
            if self.plan[0][2]:     # the first pass starts on the embedding output itself: both products in one
                z = self._mm_f32(x0, m.loop_in)
                y, y0 = z[:, :W], z[:, W:]
            else:
                y0 = self._mm_f32(x0, m.loop_in[W:])
            launches += 1
        norm1 = m.layers[self.plan[0][1]].norm1
        h = self._close(x, y, None, None, norm1, st, add=y0) if self.plan[0][2] else self._close(x, None, None, None, norm1, st)
        launches += 1
        for k, (r, li, _) in enumerate(self.plan):
            lay, rs = m.layers[li], m.run_state[r]
            la = lay.args
            o = torch.empty(n, la.mixer.heads * la.mixer.vdim, dtype=m.dtype, device=dev)
            proj = self._mm_f32(h, lay.w_in)
            launches += 2 + (self._attention if la.type == "attention" else self._latent)(lay, la, rs, proj, o, meta, st)
            y, post_w, y_bias = self._mm_f32(o, lay.w_out), lay.norm1b, lay.o_b
            if la.ff:
                h = self._close(x, y, post_w, y_bias, lay.norm2, st)
                y, c = act_unit(L, dt, h, lay.w_up, lay.w_down, None, st)
                post_w, y_bias = lay.norm2b, None
                launches += c + 1
            nxt, begins = (m.layers[self.plan[k + 1][1]].norm1, self.plan[k + 1][2]) if k + 1 < len(self.plan) else (None, False)
            if after_run is not None:       # the residual as the layer leaves it, before the next pass's product
                self._close(x, y, post_w, y_bias, None, st)
                after_run(r, x)
                y = post_w = y_bias = None
                launches += 1
                if nxt is None:
                    break
            if nxt is None and meta.all_rows:       # every row's logits are wanted: the closing kernel takes the output norm as well
                nxt = m.final_norm
            if begins:
                h = self._close(x, y, post_w, y_bias, None, st, cast=True)
                h = self._close(x, self._mm_f32(h, m.loop_in[:W]), None, None, nxt, st, add=y0)
                launches += 2
            else:
                h = self._close(x, y, post_w, y_bias, nxt, st)
            launches += 1
        self._normed = h if meta.all_rows and after_run is None else None
        self.launches = launches
        return x

    def _attention(self, lay, la, rs, proj, o, meta: StepMeta, st):
        """Softmax attention under a window -> launches."""
        L, dt, dev, tdt, a = self.L, self.dt, self.dev, self.m.dtype, la.mixer
        H, G, d, dv, n, cache = a.heads, a.kv_heads, a.dim, a.vdim, meta.n, rs.window
        qn = torch.empty(n, H, d, dtype=torch.float32, device=dev)
        kn, vn = torch.empty(n, G, d, dtype=tdt, device=dev), torch.empty(n, G, dv, dtype=tdt, device=dev)
        single = meta.seg[2] == n       # one row per sequence: the ring row it replaces has just left the window
        ring = (cache.ring, _p(cache.k), _p(cache.v)) if single else (0, None, None)
        _lib.lm_check(L.ao_lm_qkv_norm_rotary_prep(_p(proj), lay.ld, lay.q_off, lay.k_off, lay.v_off, _p(lay.q_b), _p(lay.k_b), _p(lay.v_b),
                                                   _p(lay.q_norm), _p(lay.k_norm), self.cfg.norm_eps, _p(meta.pos), _p(lay.inv_freq),
                                                   a.rot.dims, PAIR_HALVES, a.rot.amplitude, n, H, G, d, G * dv, dt, _p(qn), _p(kn), _p(vn),
                                                   _p(meta.slot), *ring, st), "qkv_norm_rotary_prep")
        c = 1 + self._window_attend(a, self._shape(la, rs), cache, qn, kn, vn, o, meta, st)
        if not single:
            self._window_append(a, cache, kn, vn, meta, st)
            c += 1
        return c

    def _latent(self, lay, la, rs, proj, o, meta: StepMeta, st):
        """Latent attention with a sink and a gate -> launches."""
        L, dt, dev, tdt, a, cache = self.L, self.dt, self.dev, self.m.dtype, la.mixer, rs.latent
        dr, R, Rq, n = a.rot_dim, a.kv_rank, a.q_rank, meta.n
        act = dict(dtype=tdt, device=dev)
        cq, c, kr = torch.empty(n, Rq, **act), torch.empty(n, R, **act), torch.empty(n, dr, **act)
        full = cache.c.shape[1] < a.window      # a cache that never wraps takes the step's rows at once
        _lib.lm_check(L.ao_lm_latent_low_prep_store(_p(proj), lay.ld, n, lay.q_off, Rq, lay.kv_off, R, dr, _p(lay.q_norm), _p(lay.c_norm), dt,
                                                    self.cfg.norm_eps, a.rot.dims, _p(lay.inv_freq), a.rot.amplitude, _p(meta.pos),
                                                    _p(meta.slot), cache.c.shape[1], _p(cq), _p(c), _p(kr), _p(cache.c) if full else None,
                                                    _p(cache.kr) if full else None, st), "latent_low_prep_store")
        shape = self._shape(la, rs)
        q, qr, k = self._latent_queries(lay, a, shape, cq, meta, st)
        launches = 1 + k + self._latent_attend(lay, a, shape, cache, c, kr, q, qr, o, meta, st, lay.sink, (proj.data_ptr() + 4 * lay.g_off, lay.ld))
        if not full:
            _lib.lm_check(L.ao_lm_ring_append(_p(c), _p(kr), n, R, dr, cache.c.shape[1], dt, _p(meta.slot), _p(meta.pos), _p(meta.ahead),
                                              _p(cache.c), _p(cache.kr), st), "ring_append")
            launches += 1
        return launches

    def _logits_dev(self, x, d_rows, k, out=None):
        m, cfg = self.m, self.cfg
        st = torch.cuda.current_stream(self.dev).cuda_stream
        xn, self._normed = self._normed, None
        if xn is None:
            xn = torch.empty(k, cfg.width, dtype=m.dtype, device=self.dev)
            _lib.lm_check(self.L.ao_lm_add_layer_norm(_p(x), None, 0.0, _p(d_rows), k, cfg.width, _p(m.final_norm), None, self.dt, cfg.norm_eps,
                                                      None, _p(xn), st), "add_layer_norm")
        return self._mm_f32(xn, m.head, out)
