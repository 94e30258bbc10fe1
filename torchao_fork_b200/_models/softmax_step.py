"""Softmax attention of the slotted sequence models whose layers are "attention" (grouped heads over a WindowKVCache) or
"latent_attention" (queries and keys through latents over a LatentKVCache), each under a sliding window or over everything
in front: the plans of both kernel forms, the tables of the expanded latent form, and the launches between a layer's
projections.  A family derives its StepEngine from SoftmaxStepEngine; its `cfg.layers[i]` carry `type` and `mixer`, its
run states `window` / `latent`.
"""
import ctypes

import numpy as np
import torch

from .. import _lib
from .products import GEMV_ROWS
from .segment_step import SegmentStepEngine, StepMeta, _p

PAIR_INTERLEAVED, PAIR_HALVES = 0, 1      # rotation couples (2i, 2i + 1) / (i, i + dims / 2)
# prompt portions attend over expanded keys and values of at most this many bytes per layer; beyond it in the folded form
EXPAND_MAX_BYTES = 4 << 30
# up to this many rows the folded form's way back is one matrix-vector kernel per head (with the gate), beyond it a batched product
VALUE_UP_ROWS = 16


class SoftmaxStepEngine(SegmentStepEngine):
    def _layer_runs(self):
        """(layer arguments, state) of every layer run; a family that runs layers more than once overrides it."""
        return list(zip(self.cfg.layers, self.m.run_state))

    # ------------------------------------------------------------------------------------------------ plans
    def _shape(self, la, ls):
        a = la.mixer
        if la.type == "attention":
            return ("window", a.heads, a.kv_heads, a.dim, a.vdim)
        return ("latent", a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, min(a.window, ls.latent.c.shape[1]))

    def _attention_shapes(self):
        return sorted({self._shape(la, ls) for la, ls in self._layer_runs() if la.type in ("attention", "latent_attention")})

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

    # ------------------------------------------------------------------------------------------------ attention
    def _window_attend(self, a, shape, cache, qn, kn, vn, row, meta: StepMeta, st):
        """Softmax of the step's queries over the ring and the step's own keys and values, into the first columns of `row`
        -> launches.  The ring is not written."""
        L, dt, dev = self.L, self.dt, self.dev
        H, G, d, dv = a.heads, a.kv_heads, a.dim, a.vdim
        tf, tc, nt, tensor = meta.attn[shape]
        window = min(a.window, cache.ring)
        common = (_p(qn), _p(kn), _p(vn), _p(cache.k), _p(cache.v), _p(cache.k_first), _p(cache.v_first), cache.ring, 0, dt, _p(meta.slot),
                  _p(meta.pos), _p(meta.back), _p(tf), _p(tc), nt, 1, H, G, d, dv, window, 0, a.scale, 0.0, 0, 0.0, 1.0)
        if tensor:      # prompt portions: the tensor-core form
            _lib.lm_check(L.ao_lm_window_attention_prompt(*common, _p(row), row.shape[1], st), "window_attention_prompt")
            return 1
        ns = self._splits(nt * G, window)    # few rows over a long window: the keys are shared out over more CTAs
        ws = torch.empty(max(16, int(L.ao_lm_window_attention_workspace_bytes(nt, 1, H, G, dv, ns))), dtype=torch.uint8, device=dev)
        _lib.lm_check(L.ao_lm_window_attention(*common, ns, _p(ws), ws.numel(), _p(row), row.shape[1], st), "window_attention")
        return 2 if ns > 1 else 1

    def _window_append(self, a, cache, kn, vn, meta: StepMeta, st):
        """The step's keys and values enter the ring, after every reader has run."""
        _lib.lm_check(self.L.ao_lm_window_append(_p(kn), _p(vn), meta.n, a.kv_heads * a.dim, a.kv_heads * a.vdim, cache.ring, 0, self.dt,
                                                 _p(meta.slot), _p(meta.pos), _p(meta.ahead), _p(cache.k), _p(cache.v), _p(cache.k_first),
                                                 _p(cache.v_first), st), "window_append")

    def _latent_queries(self, lay, a, shape, cq, meta: StepMeta, st):
        """Up-projected queries, split: -> (unrotated parts, rotated parts fp32 [n][H][dr], launches).  Unrotated parts: head-major in
        the storage type for the expanded form, multiplied by the key up-projection (fp32 [H][n][R]) for the folded one."""
        H, dn, dr, R, n = a.heads, a.dim, a.rot_dim, a.kv_rank, meta.n
        q = self._mm_f32(cq, lay.uq)
        qr = torch.empty(n, H, dr, dtype=torch.float32, device=self.dev)
        rot = (a.rot.dims, _p(lay.inv_freq), a.rot.amplitude, _p(meta.pos))
        folded = not meta.attn[shape][3]
        if folded and n <= GEMV_ROWS and self.m.dtype == torch.bfloat16 and R % 8 == 0:
            qa = torch.empty(H, n, R, dtype=torch.float32, device=self.dev)
            _lib.lm_check(self.L.ao_lm_latent_query_fold(_p(q), _p(lay.uk), self.dt, n, H, dn, dr, R, *rot, _p(qa), _p(qr), st), "latent_query_fold")
            return qa, qr, 2
        qn = torch.empty(H, n, dn, dtype=self.m.dtype, device=self.dev)
        _lib.lm_check(self.L.ao_lm_latent_query_prep(_p(q), n, H, dn, dr, self.dt, *rot, _p(qn), _p(qr), st), "latent_query_prep")
        return (self._bmm_f32(qn, lay.uk), qr, 3) if folded else (qn, qr, 2)

    def _latent_attend(self, lay, a, shape, cache, c, kr, q, qr, row, meta: StepMeta, st, sink=None, gate=None):
        """Softmax of the step's queries (as `_latent_queries` left them) over the cached latents and the step's own, into the first
        columns of `row` -> launches.  sink: a logit per head in every denominator; gate: (address, row stride) of fp32 logits per output column.
        Prompt portions attend over up-projected keys and values, few rows over the latents themselves."""
        L, dt, dev, tdt = self.L, self.dt, self.dev, self.m.dtype
        H, dn, dr, dv, R, n = a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, meta.n
        window, ring = shape[-1], cache.c.shape[1]
        tf, tc, nt, tensor = meta.attn[shape]
        g_ptr, g_ld = gate if gate is not None else (None, 0)
        if tensor:
            src, launches = meta.extra.get(("rows", window)), 2
            if src is not None:
                ca, kra = torch.empty(len(src), R, dtype=tdt, device=dev), torch.empty(len(src), dr, dtype=tdt, device=dev)
                _lib.lm_check(L.ao_lm_latent_rows_gather(_p(src), len(src), _p(c), _p(kr), _p(cache.c), _p(cache.kr), dt, R, dr, _p(ca),
                                                         _p(kra), st), "latent_rows_gather")
                c, kr, launches = ca, kra, 3
            kv = torch.mm(c, lay.ukv.t())                                              # [rows][H dn | H dv]
            ld = H * (dn + dv)
            _lib.lm_check(L.ao_lm_gated_latent_attention_expanded(
                _p(q), _p(qr), _p(kv), ld, kv.data_ptr() + kv.element_size() * H * dn, ld, _p(kr), dt, _p(meta.pos), _p(tf), _p(tc),
                _p(meta.extra[("key0", window)]), nt, n, H, dn, dr, dv, a.scale, window, _p(sink), g_ptr, g_ld, _p(row), row.shape[1], st),
                "gated_latent_attention_expanded")
            return launches
        ns = self._splits(nt * -(-H // 16), window)
        ws = torch.empty(max(16, int(L.ao_lm_latent_attention_workspace_bytes(n, H, R, ns))), dtype=torch.uint8, device=dev)
        olat = torch.empty(n, H, R, dtype=tdt, device=dev)
        _lib.lm_check(L.ao_lm_window_latent_attention(_p(q), _p(qr), _p(cache.c), _p(cache.kr), _p(c), _p(kr), dt, ring, _p(meta.slot),
                                                      _p(meta.pos), _p(meta.back), _p(tf), _p(tc), nt, n, H, R, dr, a.scale, window,
                                                      _p(sink), None, ns, _p(ws), ws.numel(), _p(olat), st), "window_latent_attention")
        launches = 2 if ns > 1 else 1
        if n <= VALUE_UP_ROWS:
            _lib.lm_check(L.ao_lm_latent_value_up(_p(olat), _p(lay.uv), dt, n, H, R, dv, g_ptr, g_ld, _p(row), row.shape[1], st),
                          "latent_value_up")
            return launches + 1
        torch.bmm(olat.transpose(0, 1), lay.uv.transpose(1, 2), out=row.as_strided((H, n, dv), (dv, row.shape[1], 1)))
        if gate is not None:
            _lib.lm_check(L.ao_lm_sigmoid_gate_rows(g_ptr, g_ld, n, H * dv, _p(row), row.shape[1], dt, st), "sigmoid_gate_rows")
            launches += 1
        return launches + 1

    def _bmm_f32(self, a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """[b][n][K] x [b][K][M] -> fp32 [b][n][M]."""
        return torch.bmm(a, w, out_dtype=torch.float32) if a.dtype == torch.bfloat16 else torch.bmm(a, w)
