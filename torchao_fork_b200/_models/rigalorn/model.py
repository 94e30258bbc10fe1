"""Rigalorn: a decoder-only language model on a pre-norm RMS residual whose two sublayers run side by side,
x += mixer(norm(x)) + ff(norm(x)) with ONE norm.  Each layer picks one of three mixers:
  * "attention": grouped heads with projection biases under a sliding window; rotation of the first coordinates (pairs
    (i, i + dims/2)), optionally with YaRN scaling; layers that mix values add a learned share of the first such layer's
    values of the same token to their own before they are cached;
  * "delta": gated delta rule over a matrix state per head; queries, keys and values pass short causal convolutions and SiLU,
    queries and keys are unit vectors; every head's read-out is brought to unit RMS, weighted and gated by SiLU;
  * "latent_attention": queries, keys and values through latents, one rotated key part shared by all heads (pairs
    (2i, 2i + 1)), under a sliding window; only the latent and the rotated key part are cached.
The feed-forward is W_down xIELU(W_up h); a layer may have none.

Because both sublayers read one row and add into one row, a layer is two large products: every projection of the mixer and
the feed-forward's up-projection are ONE operand, and so are the mixer's output projection and the down-projection.

This module holds the configuration (every size and constant is read from a checkpoint's config.json or from a tensor's
shape), the weights in the layout the kernels want, and the per-sequence state (cache.py).  The compute is step.py.
Checkpoint tensor names: embed, final.norm, head, l<i>.norm1, l<i>.mix.{q,k,v}[.b], l<i>.mix.{vmix,o} |
l<i>.mix.{q,k,v}[.conv], l<i>.mix.{a,b,g,A_log,dt_bias,norm,o} | l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o},
l<i>.mlp.{up,down,act}; linear weights are [out][in].
"""
import math
import os
import warnings
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch
import torch.nn as nn

from ..cache import ConvState, LatentKVCache, MatrixState, SequenceStates, WindowKVCache
from ..checkpoint import read_config, read_safetensors
from ..rotary import RotaryArgs, RotaryScaling

NO_WINDOW = 1 << 30     # a mask without a window size: plain causal attention
UNIT_EPS = 1e-6         # of the delta rule's unit queries and keys


@dataclass
class AttentionArgs:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = NO_WINDOW
    rot: RotaryArgs = field(default_factory=RotaryArgs)
    v_mix: bool = False


@dataclass
class DeltaArgs:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @property
    def channels(self):         # of the convolutions: [queries | keys | values]
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def padded_dim(self):       # key entries per row of the state: whole 16-byte pieces
        return -(-self.dim // 4) * 4


@dataclass
class LatentAttentionArgs:
    heads: int
    dim: int                    # unrotated query / key size per head
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int = NO_WINDOW
    rot: RotaryArgs = field(default_factory=RotaryArgs)


@dataclass
class LayerArgs:
    type: str                   # "attention" | "delta" | "latent_attention"
    mixer: object
    ff: int = 0                 # 0: no feed-forward


def _window(m) -> int:
    size = (m.get("mask") or {}).get("size")
    return NO_WINDOW if size is None else int(size)


@dataclass
class RigalornArgs:
    vocab_size: int
    width: int
    norm_eps: float
    embedding_scale: float = 1.0
    layers: List[LayerArgs] = field(default_factory=list)
    block_size: int = 1 << 30

    @property
    def n_layer(self):
        return len(self.layers)

    @property
    def first_v_mix(self) -> Optional[int]:
        """The layer whose values the other value-mixing layers add to their own."""
        return next((i for i, la in enumerate(self.layers) if la.type == "attention" and la.mixer.v_mix), None)

    @classmethod
    def from_dict(cls, cfg: dict) -> "RigalornArgs":
        layers = []
        for i, lay in enumerate(cfg["layers"]):
            m, kind = lay["mixer"], lay["type"]
            if kind == "attention":
                mixer = AttentionArgs(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), _window(m),
                                      RotaryArgs.from_dict(m.get("rot")), bool(m.get("v_mix", False)))
                assert mixer.heads % mixer.kv_heads == 0, f"layer {i}: {mixer.heads} heads over {mixer.kv_heads} key/value heads"
                assert mixer.rot.dims % 2 == 0 and 0 <= mixer.rot.dims <= mixer.dim, f"layer {i}: rotation over {mixer.rot.dims} of {mixer.dim}"
                assert mixer.vdim <= 256, f"layer {i}: the window attention kernel keeps at most 256 values per head"
            elif kind == "delta":
                mixer = DeltaArgs(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
                assert mixer.heads % mixer.kv_heads == 0, f"layer {i}: {mixer.heads} heads over {mixer.kv_heads} query/key heads"
                assert mixer.taps >= 1 and mixer.dim <= 1024, f"layer {i}: {mixer}"
            elif kind == "latent_attention":
                mixer = LatentAttentionArgs(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["q_rank"]),
                                            int(m["kv_rank"]), float(m["scale"]), _window(m), RotaryArgs.from_dict(m.get("rot")))
                assert mixer.rot.dims % 2 == 0 and mixer.rot.dims <= mixer.rot_dim, f"layer {i}: rotation over {mixer.rot.dims} of {mixer.rot_dim}"
                assert mixer.kv_rank <= 512, f"layer {i}: the latent attention kernels keep at most 512 latent values"
            else:
                raise NotImplementedError(f"layer {i}: mixer type {kind!r}")
            assert kind == "delta" or mixer.window >= 1, f"layer {i}: a window of {mixer.window}"
            f, ff = lay.get("mlp"), 0
            if f:
                if f.get("kind", "dense") != "dense":
                    raise NotImplementedError(f"layer {i}: feed-forward kind {f['kind']!r}")
                ff = int(f["ff"])
            layers.append(LayerArgs(kind, mixer, ff))
        self = cls(vocab_size=int(cfg["vocab"]), width=int(cfg["width"]), norm_eps=float(cfg["norm"]["eps"]),
                   embedding_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)), layers=layers)
        j = self.first_v_mix
        for i, la in enumerate(layers):
            if la.type == "attention" and la.mixer.v_mix:
                a, b = la.mixer, layers[j].mixer
                assert a.kv_heads * a.vdim == b.kv_heads * b.vdim, f"layer {i} mixes in layer {j}'s values, which have another size"
        return self

    def to_dict(self) -> dict:
        out = []
        for la in self.layers:
            m = la.mixer
            if la.type == "attention":
                mx = {"dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads, "scale": m.scale, "vdim": m.vdim}
                if m.v_mix:
                    mx["v_mix"] = True
            elif la.type == "delta":
                mx = {"conv": m.taps, "dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads, "vdim": m.vdim}
            else:
                mx = {"dim": m.dim, "heads": m.heads, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "rot_dim": m.rot_dim, "scale": m.scale,
                      "vdim": m.vdim}
            if la.type != "delta":
                if m.window != NO_WINDOW:
                    mx["mask"] = {"size": m.window}
                if m.rot.dims:
                    mx["rot"] = m.rot.to_dict()
            out.append({"mixer": mx, "mlp": {"ff": la.ff, "kind": "dense"} if la.ff else None, "type": la.type})
        return {"architecture": "Rigalorn", "embedding": {"scale": self.embedding_scale}, "layers": out, "norm": {"eps": self.norm_eps},
                "vocab": self.vocab_size, "width": self.width}


def _pattern(n_layer, width, heads, kv_heads, dim, ff, vocab, window=4096, q_rank=768, kv_rank=512, rot_dim=64, taps=4):
    """Layers cycling latent attention -> attention -> delta."""
    layers = []
    for i in range(n_layer):
        kind = ("latent_attention", "attention", "delta")[i % 3]
        if kind == "latent_attention":
            mixer = LatentAttentionArgs(heads, dim, rot_dim, dim, q_rank, kv_rank, 1.0 / math.sqrt(dim + rot_dim), window,
                                        RotaryArgs(rot_dim, 5e5))
        elif kind == "attention":
            mixer = AttentionArgs(heads, kv_heads, dim, dim, 1.0 / math.sqrt(dim), window,
                                  RotaryArgs(dim // 2, 1e6, RotaryScaling(8.0, 4096.0, 32.0, 1.0)), True)
        else:
            mixer = DeltaArgs(heads, max(1, heads // 2), dim, dim, taps)
        layers.append(LayerArgs(kind, mixer, ff))
    return RigalornArgs(vocab, width, 1e-6, 1.0, layers)


# named random-init configurations (benchmarks and examples; checkpoints carry their own config.json)
rigalorn_configs = {
    "Rigalorn-test": lambda: _pattern(6, 128, 4, 2, 32, 320, 512, window=24, q_rank=48, kv_rank=64, rot_dim=16),
    # layers of the size of a 1-2 B parameter model / of a 7-8 B parameter model (a layer benchmark); an ungated feed-forward of
    # 4.5 widths holds as many weights as a gated one of 3 widths
    "Rigalorn-2k": lambda: _pattern(3, 2048, 16, 4, 128, 9216, 32000),
    "Rigalorn-4k": lambda: _pattern(3, 4096, 32, 8, 128, 18432, 128256, q_rank=1536),
}


class _Layer:
    """One layer's tensors as the kernels read them (plain attributes; the module registers them as buffers)."""


class _LayerState:
    """Per-sequence state of one layer."""
    window: Optional[WindowKVCache] = None
    latent: Optional[LatentKVCache] = None
    mat: Optional[MatrixState] = None
    conv: Optional[ConvState] = None

    def parts(self):
        return [p for p in (self.window, self.latent, self.mat, self.conv) if p is not None]


class Rigalorn(nn.Module):
    def __init__(self, config: RigalornArgs, weights: Dict[str, torch.Tensor], device="cuda", dtype=torch.bfloat16):
        super().__init__()
        assert dtype in (torch.bfloat16, torch.float32), "Rigalorn runs in bfloat16 or float32"
        self.config, self.dtype = config, dtype
        self.device = torch.device(device)
        self.max_batch_size = -1
        self.max_seq_length = -1
        self.states: Optional[SequenceStates] = None
        self.run_state: List[_LayerState] = []
        self._step = None
        self._take(weights)

    # ------------------------------------------------------------------------------------------------ weights
    def _take(self, w: Dict[str, torch.Tensor]):
        cfg, dev, dt = self.config, self.device, self.dtype
        used = set()

        def get(name, shape=None, dtype=dt):
            if name not in w:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            used.add(name)
            t = w[name]
            if shape is not None and tuple(t.shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration asks for {tuple(shape)}")
            return t.to(device=dev, dtype=dtype)

        def buf(name, t):
            self.register_buffer(name.replace(".", "__"), t.contiguous(), persistent=False)
            return getattr(self, name.replace(".", "__"))

        def stack(*named):      # rows of one projection operand -> (the operand, tensor name -> its first row)
            at, offs = 0, {}
            for name, rows in named:
                offs[name] = at
                at += rows
            return torch.cat([get(name, (rows, W)) for name, rows in named], 0), offs

        W, V = cfg.width, cfg.vocab_size
        self.embed = buf("embed", get("embed", (V, W)))
        self.final_norm = buf("final.norm", get("final.norm", (W,)))
        self.head = buf("head", get("head", (V, W)))
        self.layers: List[_Layer] = []
        for i, la in enumerate(cfg.layers):
            q, L, m, ff = f"l{i}.mix.", _Layer(), la.mixer, la.ff
            L.args = la
            L.norm1 = buf(f"l{i}.norm1", get(f"l{i}.norm1", (W,)))
            up = [(f"l{i}.mlp.up", ff)] if ff else []
            H = m.heads
            if la.type == "attention":
                G, d, dv = m.kv_heads, m.dim, m.vdim
                w_in, offs = stack((q + "q", H * d), (q + "k", G * d), (q + "v", G * dv), *up)
                L.q_off, L.k_off, L.v_off = (offs[q + s] for s in "qkv")
                L.q_b, L.k_b, L.v_b = (buf(q + s + ".b", get(q + s + ".b", (n,))) for s, n in (("q", H * d), ("k", G * d), ("v", G * dv)))
                L.lam = float(get(q + "vmix", None, torch.float64).reshape(())) if m.v_mix else 0.0
            elif la.type == "delta":
                G, d, dv, C = m.kv_heads, m.dim, m.vdim, m.channels
                w_in, offs = stack((q + "q", G * d), (q + "k", G * d), (q + "v", H * dv), (q + "g", H * dv), *up, (q + "a", H), (q + "b", H))
                L.g_off, L.a_off, L.b_off = (offs[q + s] for s in "gab")
                kernels = torch.cat([get(q + s + ".conv", (n, m.taps)) for s, n in (("q", G * d), ("k", G * d), ("v", H * dv))], 0)
                L.conv_w = buf(q + "conv", kernels.t())                                     # [taps][channels]
                L.a_log, L.dt_bias = buf(q + "A_log", get(q + "A_log", (H,))), buf(q + "dt_bias", get(q + "dt_bias", (H,)))
                L.mix_norm = buf(q + "norm", get(q + "norm", (dv,)))
            else:
                dn, dr, dv, R, Rq = m.dim, m.rot_dim, m.vdim, m.kv_rank, m.q_rank
                w_in, offs = stack((q + "dq", Rq), (q + "dkv", R + dr), *up)
                L.q_off, L.kv_off = offs[q + "dq"], offs[q + "dkv"]
                L.q_norm, L.c_norm = buf(q + "dq.norm", get(q + "dq.norm", (Rq,))), buf(q + "dkv.norm", get(q + "dkv.norm", (R,)))
                L.uq = buf(q + "uq", get(q + "uq", (H * (dn + dr), Rq)))
                # keys and values of all heads as one operand (prompt portions); per head for the folded form (decoded tokens)
                L.ukv = buf(q + "ukv", torch.cat([get(q + "uk", (H * dn, R)), get(q + "uv", (H * dv, R))], 0))
                L.uk = L.ukv[: H * dn].view(H, dn, R)
                L.uv = L.ukv[H * dn:].view(H, dv, R)
            if la.type != "delta":
                L.inv_freq = buf(q + "inv_freq", m.rot.inv_freq(dev)) if m.rot.dims else None
            L.w_in, L.ld = buf(q + "in", w_in), w_in.shape[0]
            L.o_width = H * m.vdim
            out = [get(q + "o", (W, L.o_width))]
            if ff:
                r = f"l{i}.mlp."
                L.up_off = offs[r + "up"]
                out.append(get(r + "down", (W, ff)))
                p = torch.nn.functional.softplus(get(r + "act", (2,), torch.float64), threshold=1e9).tolist()
                L.act_pos, L.act_neg = p[0], 0.5 + p[1]
            L.w_out = buf(q + "out", torch.cat(out, 1))
            self.layers.append(L)
        extra = sorted(set(w) - used)
        if extra:   # e.g. the value share of a layer that mixes nothing: nothing reads it
            warnings.warn(f"checkpoint tensors the configuration does not use: {extra[:8]}{' ...' if len(extra) > 8 else ''}")

    @classmethod
    def from_checkpoint(cls, folder, device="cuda", dtype=torch.bfloat16):
        w = read_safetensors(os.path.join(str(folder), "model.safetensors"))
        return cls(RigalornArgs.from_dict(read_config(folder)), w, device, dtype).eval()

    @classmethod
    def from_name(cls, name, device="cuda", dtype=torch.bfloat16):
        return cls.random_init(rigalorn_configs[name](), device, dtype)

    @staticmethod
    def random_weights(cfg: RigalornArgs, device="cpu", dtype=torch.bfloat16, seed=1234) -> Dict[str, torch.Tensor]:
        """Seeded random weights of every tensor the configuration names (no checkpoints exist offline)."""
        g = torch.Generator(device=device).manual_seed(seed)
        W = cfg.width

        def mat(o, i, s=1.0):
            return (torch.randn(o, i, generator=g, device=device, dtype=torch.float32) * (s / math.sqrt(i))).to(dtype)

        def vec(n, mean=0.0, s=1.0):
            n = n if isinstance(n, tuple) else (n,)
            return (mean + s * torch.randn(*n, generator=g, device=device, dtype=torch.float32)).to(dtype)

        w = {"embed": vec((cfg.vocab_size, W), 0.0, 1.0), "head": mat(cfg.vocab_size, W), "final.norm": vec(W, 1.0, 0.1)}
        for i, la in enumerate(cfg.layers):
            q, m = f"l{i}.mix.", la.mixer
            w[f"l{i}.norm1"] = vec(W, 1.0, 0.1)
            H, dv = m.heads, m.vdim
            if la.type == "attention":
                for s, n in (("q", H * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * dv)):
                    w[q + s], w[q + s + ".b"] = mat(n, W), vec(n, 0.0, 0.2)
                if m.v_mix:
                    w[q + "vmix"] = torch.tensor(0.3, dtype=dtype, device=device)
            elif la.type == "delta":
                for s, n in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", H * dv)):
                    w[q + s], w[q + s + ".conv"] = mat(n, W), vec((n, m.taps), 0.2, 0.4)
                w[q + "g"], w[q + "a"], w[q + "b"] = mat(H * dv, W), mat(H, W), mat(H, W)
                w[q + "A_log"], w[q + "dt_bias"], w[q + "norm"] = vec(H, -1.0, 1.0), vec(H, -2.0, 1.0), vec(dv, 1.0, 0.1)
            else:
                w[q + "dq"], w[q + "dq.norm"], w[q + "uq"] = mat(m.q_rank, W), vec(m.q_rank, 1.0, 0.1), mat(H * (m.dim + m.rot_dim), m.q_rank)
                w[q + "dkv"], w[q + "dkv.norm"] = mat(m.kv_rank + m.rot_dim, W), vec(m.kv_rank, 1.0, 0.1)
                w[q + "uk"], w[q + "uv"] = mat(H * m.dim, m.kv_rank), mat(H * dv, m.kv_rank)
            w[q + "o"] = mat(W, H * dv)
            if la.ff:
                r = f"l{i}.mlp."
                w[r + "up"], w[r + "down"], w[r + "act"] = mat(la.ff, W), mat(W, la.ff), vec(2, 0.0, 0.3)
        return w

    @classmethod
    def random_init(cls, cfg: RigalornArgs, device="cuda", dtype=torch.bfloat16, seed=1234):
        return cls(cfg, cls.random_weights(cfg, device, dtype, seed), device, dtype).eval()

    def weight_bytes(self, ignore_embeddings=False) -> int:
        skip = {"embed"} if ignore_embeddings else set()
        return sum(b.numel() * b.element_size() for n, b in self.named_buffers() if n not in skip)

    # ------------------------------------------------------------------------------------------------ state
    def setup_caches(self, max_batch_size, max_seq_length, dtype=None, device=None, kv_cache_quantization=False):
        """Per-sequence state for `max_batch_size` slots: a ring as long as the window (never longer than max_seq_length) of
        keys and values (attention) or of latents and rotated key parts (latent attention); a matrix state per head and the
        convolutions' last inputs (delta).  A sequence may grow past max_seq_length when no window had to be cut to it.  Same
        call as the Llama's setup_caches."""
        if kv_cache_quantization:
            raise NotImplementedError("Rigalorn keeps its keys, values and latents in the model's dtype")
        if self.states is not None and self.max_seq_length >= max_seq_length and self.max_batch_size >= max_batch_size:
            return
        cfg, dev, n = self.config, self.device, max_batch_size
        self.max_batch_size, self.max_seq_length = max_batch_size, max_seq_length
        self.run_state = []
        bounded = False
        for la in cfg.layers:
            m, ls = la.mixer, _LayerState()
            if la.type == "delta":
                ls.mat = MatrixState(n, m.heads, m.vdim, m.padded_dim, dev)      # a value column's entries are neighbours
                ls.conv = ConvState(n, m.taps, m.channels, dev)
            else:
                bounded |= m.window > max_seq_length
                ring = min(m.window, max_seq_length)
                if la.type == "attention":
                    ls.window = WindowKVCache(n, ring, 0, m.kv_heads * m.dim, m.kv_heads * m.vdim, self.dtype, dev)
                else:
                    ls.latent = LatentKVCache(n, ring, m.kv_rank, m.rot_dim, self.dtype, dev)
            self.run_state.append(ls)
        self.states = SequenceStates(n, max_seq_length if bounded else 1 << 30)
        for ls in self.run_state:
            for part in ls.parts():
                self.states.on_grow.append(part.grow)
        self.states.on_grow.append(lambda k: setattr(self, "max_batch_size", k))
        self._step = None

    def state_bytes_per_sequence(self) -> int:
        return sum(b.numel() * b.element_size() for ls in self.run_state for part in ls.parts() for b in part.buffers()) \
            // self.max_batch_size

    @property
    def step_engine(self):
        """The step function over this model's weights and state (step.py), made on first use."""
        if self._step is None:
            from .step import StepEngine
            assert self.states is not None, "call setup_caches first"
            self._step = StepEngine(self)
        return self._step

    def make_decode_engine(self, batch_size, temperature=0.8, top_k=200, **unused):
        from .step import GraphDecodeEngine
        return GraphDecodeEngine(self, batch_size, temperature, top_k)

    @torch.no_grad()
    def forward(self, idx: torch.Tensor, input_pos: Optional[torch.Tensor] = None) -> torch.Tensor:
        """idx [B][T] at positions input_pos [T] (default 0 .. T-1) of the sequences in slots 0 .. B-1 -> logits of the
        LAST position [B][1][vocab] in fp32 (what generation samples from).  The Llama's forward call shape.  The state
        is recurrent: positions must continue where the slots stand (or restart at 0)."""
        assert self.states is not None, "Caches must be initialized first"
        B, T = idx.shape
        start = 0 if input_pos is None else int(input_pos[0])
        st = self.states
        segs = []
        for b in range(B):
            slot = st.slot_of(("batch", b))
            assert slot == b, "generation batches own slots 0 .. B-1: release other requests first"
            assert start == 0 or st.length[slot] == start, "a recurrent state cannot jump to another position"
            st.length[slot] = start
            segs.append((slot, idx[b]))
        logits = self.step_engine.step(segs, want="last")
        return logits.view(B, 1, -1)
