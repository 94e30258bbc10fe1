"""Sozanex: a decoder-only language model with a layer norm (a weight, no bias) in front of and behind every sublayer,
x += norm1b(mixer(norm1(x))), x += norm2b(ff(norm2(x))).  Each layer picks one of two mixers:
  * "attention": grouped heads with projection biases, RMS-normed queries and keys (one weight for all heads), rotation of the
    first coordinates (pairs (i, i + dims/2)), optionally with band scaling, under a sliding window;
  * "latent_attention": queries, keys and values through latents, one rotated key part shared by all heads (pairs
    (2i, 2i + 1)), optionally with YaRN scaling; causal over everything in front, a sink logit per head in the softmax
    denominator, the concatenated heads times the sigmoid of a projection of their own; only the latent and the rotated key
    part are cached.
The feed-forward is W_down relu(W_up h)^2; a layer may have none.  The embedding adds a row of a hashed table of (previous token,
token) pairs.  A span of layers may run several times with the same weights; in front of every pass the residual becomes
W_in [x; embedding output], and every pass keeps a state of its own.

This module holds the configuration (every size and constant is read from a checkpoint's config.json or from a tensor's
shape), the weights in the layout the kernels want, and the per-sequence state (cache.py).  The compute is step.py.
Checkpoint tensor names: embed, bigram, loop.in, final.norm, head, l<i>.norm{1,1b,2,2b},
l<i>.mix.{q,k,v,o}[.b], l<i>.mix.{q,k}.norm | l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,g,o}, l<i>.mlp.{up,down}; linear
weights are [out][in].
"""
import math
import os
import warnings
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..cache import LastTokenState, LatentKVCache, SequenceStates, WindowKVCache
from ..checkpoint import read_config, read_safetensors
from ..rotary import BandScaling, RotaryArgs, RotaryScaling

NO_WINDOW = 1 << 30     # a mask without a window size: plain causal attention


@dataclass
class AttentionArgs:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = NO_WINDOW
    rot: RotaryArgs = field(default_factory=RotaryArgs)


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
    type: str                   # "attention" | "latent_attention"
    mixer: object
    ff: int = 0                 # 0: no feed-forward


@dataclass
class BigramArgs:
    buckets: int
    mul_prev: int
    mul_cur: int


def _window(m) -> int:
    size = (m.get("mask") or {}).get("size")
    return NO_WINDOW if size is None else int(size)


@dataclass
class SozanexArgs:
    vocab_size: int
    width: int
    norm_eps: float
    embedding_scale: float = 1.0
    bigram: Optional[BigramArgs] = None
    loop: Optional[Tuple[int, int, int]] = None     # (start, stop, times)
    layers: List[LayerArgs] = field(default_factory=list)
    block_size: int = 1 << 30

    @property
    def n_layer(self):
        return len(self.layers)

    @property
    def schedule(self) -> List[Tuple[int, bool]]:
        """(layer index, does a pass begin in front of it) of every layer run, in order."""
        n = len(self.layers)
        if not self.loop:
            return [(i, False) for i in range(n)]
        a, b, times = self.loop
        return [(i, False) for i in range(a)] + [(i, i == a) for i in range(a, b)] * times + [(i, False) for i in range(b, n)]

    @property
    def runs(self) -> List[int]:
        """Layer index of every layer run, in order (a looped layer appears once per pass)."""
        return [i for i, _ in self.schedule]

    @classmethod
    def from_dict(cls, cfg: dict) -> "SozanexArgs":
        layers = []
        for i, lay in enumerate(cfg["layers"]):
            m, kind = lay["mixer"], lay["type"]
            if kind == "attention":
                mixer = AttentionArgs(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), _window(m),
                                      RotaryArgs.from_dict(m.get("rot")))
                assert mixer.heads % mixer.kv_heads == 0, f"layer {i}: {mixer.heads} heads over {mixer.kv_heads} key/value heads"
                assert mixer.rot.dims % 2 == 0 and 0 <= mixer.rot.dims <= mixer.dim, f"layer {i}: rotation over {mixer.rot.dims} of {mixer.dim}"
                assert mixer.vdim <= 256, f"layer {i}: the window attention kernel keeps at most 256 values per head"
            elif kind == "latent_attention":
                mixer = LatentAttentionArgs(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["q_rank"]),
                                            int(m["kv_rank"]), float(m["scale"]), _window(m), RotaryArgs.from_dict(m.get("rot")))
                assert mixer.rot.dims % 2 == 0 and mixer.rot.dims <= mixer.rot_dim, f"layer {i}: rotation over {mixer.rot.dims} of {mixer.rot_dim}"
                assert mixer.kv_rank <= 512, f"layer {i}: the latent attention kernels keep at most 512 latent values"
            else:
                raise NotImplementedError(f"layer {i}: mixer type {kind!r}")
            assert mixer.window >= 1, f"layer {i}: a window of {mixer.window}"
            f, ff = lay.get("mlp"), 0
            if f:
                if f.get("kind", "dense") != "dense":
                    raise NotImplementedError(f"layer {i}: feed-forward kind {f['kind']!r}")
                ff = int(f["ff"])
            layers.append(LayerArgs(kind, mixer, ff))
        loop = cfg.get("loop")
        if loop:
            loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
            assert 0 <= loop[0] < loop[1] <= len(layers) and loop[2] >= 1, f"loop {loop} over {len(layers)} layers"
        e = cfg.get("embedding") or {}
        b = e.get("bigram")
        return cls(vocab_size=int(cfg["vocab"]), width=int(cfg["width"]), norm_eps=float(cfg["norm"]["eps"]),
                   embedding_scale=float(e.get("scale", 1.0)),
                   bigram=BigramArgs(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b else None, loop=loop or None, layers=layers)

    def to_dict(self) -> dict:
        out = []
        for la in self.layers:
            m = la.mixer
            if la.type == "attention":
                mx = {"dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads, "scale": m.scale, "vdim": m.vdim}
            else:
                mx = {"dim": m.dim, "heads": m.heads, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "rot_dim": m.rot_dim, "scale": m.scale,
                      "vdim": m.vdim}
            if m.window != NO_WINDOW:
                mx["mask"] = {"size": m.window}
            if m.rot.dims:
                mx["rot"] = m.rot.to_dict()
            out.append({"mixer": mx, "mlp": {"ff": la.ff, "kind": "dense"} if la.ff else None, "type": la.type})
        e = {"scale": self.embedding_scale}
        if self.bigram:
            e["bigram"] = {"buckets": self.bigram.buckets, "mul_cur": self.bigram.mul_cur, "mul_prev": self.bigram.mul_prev}
        cfg = {"architecture": "Sozanex", "embedding": e, "layers": out, "norm": {"eps": self.norm_eps}, "vocab": self.vocab_size,
               "width": self.width}
        if self.loop:
            cfg["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return cfg


def _pattern(n_layer, width, heads, kv_heads, dim, ff, vocab, window=4096, q_rank=768, kv_rank=512, rot_dim=64, loop=None, buckets=65521):
    """Layers cycling latent attention -> attention."""
    layers = []
    for i in range(n_layer):
        if i % 2 == 0:
            mixer = LatentAttentionArgs(heads, dim, rot_dim, dim, q_rank, kv_rank, 1.0 / math.sqrt(dim + rot_dim), NO_WINDOW,
                                        RotaryArgs(rot_dim, 5e5, RotaryScaling(8.0, 4096.0, 32.0, 1.0)))
        else:
            mixer = AttentionArgs(heads, kv_heads, dim, dim, 1.0 / math.sqrt(dim), window,
                                  RotaryArgs(dim // 2, 1e6, BandScaling(8.0, 8192.0, 1.0, 4.0)))
        layers.append(LayerArgs("attention" if i % 2 else "latent_attention", mixer, ff))
    return SozanexArgs(vocab, width, 1e-6, 1.0, BigramArgs(buckets, 31337, 7919), loop, layers)


# named random-init configurations (benchmarks and examples; checkpoints carry their own config.json)
sozanex_configs = {
    "Sozanex-test": lambda: _pattern(4, 128, 4, 2, 32, 320, 512, window=24, q_rank=48, kv_rank=64, rot_dim=16, loop=(1, 3, 2), buckets=509),
    # layers of the size of a 1-2 B parameter model / of a 7-8 B parameter model (a layer benchmark); an ungated feed-forward of
    # 4.5 widths holds as many weights as a gated one of 3 widths
    "Sozanex-2k": lambda: _pattern(2, 2048, 16, 4, 128, 9216, 32000),
    "Sozanex-4k": lambda: _pattern(2, 4096, 32, 8, 128, 18432, 128256, q_rank=1536),
    # the same layers run twice over
    "Sozanex-2k-loop": lambda: _pattern(2, 2048, 16, 4, 128, 9216, 32000, loop=(0, 2, 2)),
}


class _Layer:
    """One layer's tensors as the kernels read them (plain attributes; the module registers them as buffers)."""


class _RunState:
    """Per-sequence state of ONE layer run (a looped layer has one per pass), or of the embedding."""
    window: Optional[WindowKVCache] = None
    latent: Optional[LatentKVCache] = None
    last: Optional[LastTokenState] = None

    def parts(self):
        return [p for p in (self.window, self.latent, self.last) if p is not None]


class Sozanex(nn.Module):
    def __init__(self, config: SozanexArgs, weights: Dict[str, torch.Tensor], device="cuda", dtype=torch.bfloat16):
        super().__init__()
        assert dtype in (torch.bfloat16, torch.float32), "Sozanex runs in bfloat16 or float32"
        self.config, self.dtype = config, dtype
        self.device = torch.device(device)
        self.max_batch_size = -1
        self.max_seq_length = -1
        self.states: Optional[SequenceStates] = None
        self.run_state: List[_RunState] = []        # one per layer run; the embedding's, when it has one, comes last
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
        self.bigram = buf("bigram", get("bigram", (cfg.bigram.buckets + 1, W))) if cfg.bigram else None
        self.final_norm = buf("final.norm", get("final.norm", (W,)))
        self.head = buf("head", get("head", (V, W)))
        if cfg.loop:    # W_in [x; x0] as two products: rows for the residual, then rows for the embedding output
            w_in = get("loop.in", (W, 2 * W))
            self.loop_in = buf("loop.in", torch.cat([w_in[:, :W], w_in[:, W:]], 0))
        self.layers: List[_Layer] = []
        for i, la in enumerate(cfg.layers):
            p, q, L, m, ff = f"l{i}.", f"l{i}.mix.", _Layer(), la.mixer, la.ff
            L.args = la
            L.norm1, L.norm1b = buf(p + "norm1", get(p + "norm1", (W,))), buf(p + "norm1b", get(p + "norm1b", (W,)))
            H = m.heads
            if la.type == "attention":
                G, d, dv = m.kv_heads, m.dim, m.vdim
                w_in, offs = stack((q + "q", H * d), (q + "k", G * d), (q + "v", G * dv))
                L.q_off, L.k_off, L.v_off = (offs[q + s] for s in "qkv")
                L.q_b, L.k_b, L.v_b = (buf(q + s + ".b", get(q + s + ".b", (n,))) for s, n in (("q", H * d), ("k", G * d), ("v", G * dv)))
                L.q_norm, L.k_norm = buf(q + "q.norm", get(q + "q.norm", (d,))), buf(q + "k.norm", get(q + "k.norm", (d,)))
                L.o_b = buf(q + "o.b", get(q + "o.b", (W,), torch.float32))           # added to the fp32 product
            else:
                dn, dr, dv, R, Rq = m.dim, m.rot_dim, m.vdim, m.kv_rank, m.q_rank
                w_in, offs = stack((q + "g", H * dv), (q + "dq", Rq), (q + "dkv", R + dr))
                L.g_off, L.q_off, L.kv_off = offs[q + "g"], offs[q + "dq"], offs[q + "dkv"]
                L.q_norm, L.c_norm = buf(q + "dq.norm", get(q + "dq.norm", (Rq,))), buf(q + "dkv.norm", get(q + "dkv.norm", (R,)))
                L.uq = buf(q + "uq", get(q + "uq", (H * (dn + dr), Rq)))
                # keys and values of all heads as one operand (prompt portions); per head for the folded form (decoded tokens)
                L.ukv = buf(q + "ukv", torch.cat([get(q + "uk", (H * dn, R)), get(q + "uv", (H * dv, R))], 0))
                L.uk = L.ukv[: H * dn].view(H, dn, R)
                L.uv = L.ukv[H * dn:].view(H, dv, R)
                L.sink = buf(q + "sink", get(q + "sink", (H,)))
                L.o_b = None
            L.inv_freq = buf(q + "inv_freq", m.rot.inv_freq(dev)) if m.rot.dims else None
            L.w_in, L.ld = buf(q + "in", w_in), w_in.shape[0]
            L.w_out = buf(q + "o", get(q + "o", (W, H * m.vdim)))
            if ff:
                L.norm2, L.norm2b = buf(p + "norm2", get(p + "norm2", (W,))), buf(p + "norm2b", get(p + "norm2b", (W,)))
                L.w_up, L.w_down = buf(p + "mlp.up", get(p + "mlp.up", (ff, W))), buf(p + "mlp.down", get(p + "mlp.down", (W, ff)))
            self.layers.append(L)
        extra = sorted(set(w) - used)
        if extra:   # e.g. the feed-forward norms of a layer that has no feed-forward: nothing reads them
            warnings.warn(f"checkpoint tensors the configuration does not use: {extra[:8]}{' ...' if len(extra) > 8 else ''}")

    @classmethod
    def from_checkpoint(cls, folder, device="cuda", dtype=torch.bfloat16):
        w = read_safetensors(os.path.join(str(folder), "model.safetensors"))
        return cls(SozanexArgs.from_dict(read_config(folder)), w, device, dtype).eval()

    @classmethod
    def from_name(cls, name, device="cuda", dtype=torch.bfloat16):
        return cls.random_init(sozanex_configs[name](), device, dtype)

    @staticmethod
    def random_weights(cfg: SozanexArgs, device="cpu", dtype=torch.bfloat16, seed=1234) -> Dict[str, torch.Tensor]:
        """Seeded random weights of every tensor the configuration names (no checkpoints exist offline)."""
        g = torch.Generator(device=device).manual_seed(seed)
        W = cfg.width

        def mat(o, i, s=1.0):
            return (torch.randn(o, i, generator=g, device=device, dtype=torch.float32) * (s / math.sqrt(i))).to(dtype)

        def vec(n, mean=0.0, s=1.0):
            return (mean + s * torch.randn(n, generator=g, device=device, dtype=torch.float32)).to(dtype)

        w = {"embed": mat(cfg.vocab_size, W, math.sqrt(W)), "head": mat(cfg.vocab_size, W), "final.norm": vec(W, 1.0, 0.1)}
        if cfg.bigram:
            w["bigram"] = mat(cfg.bigram.buckets + 1, W, 0.5 * math.sqrt(W))
        if cfg.loop:
            w["loop.in"] = mat(W, 2 * W)
        for i, la in enumerate(cfg.layers):
            p, q, m = f"l{i}.", f"l{i}.mix.", la.mixer
            w[p + "norm1"], w[p + "norm1b"] = vec(W, 1.0, 0.1), vec(W, 1.0, 0.1)
            H, dv = m.heads, m.vdim
            if la.type == "attention":
                for s, n in (("q", H * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * dv)):
                    w[q + s], w[q + s + ".b"] = mat(n, W), vec(n, 0.0, 0.2)
                w[q + "q.norm"], w[q + "k.norm"], w[q + "o.b"] = vec(m.dim, 1.0, 0.1), vec(m.dim, 1.0, 0.1), vec(W, 0.0, 0.2)
            else:
                w[q + "dq"], w[q + "dq.norm"], w[q + "uq"] = mat(m.q_rank, W), vec(m.q_rank, 1.0, 0.1), mat(H * (m.dim + m.rot_dim), m.q_rank)
                w[q + "dkv"], w[q + "dkv.norm"] = mat(m.kv_rank + m.rot_dim, W), vec(m.kv_rank, 1.0, 0.1)
                w[q + "uk"], w[q + "uv"] = mat(H * m.dim, m.kv_rank), mat(H * dv, m.kv_rank)
                w[q + "sink"], w[q + "g"] = vec(H, 0.0, 1.0), mat(H * dv, W)
            w[q + "o"] = mat(W, H * dv)
            if la.ff:
                w[p + "norm2"], w[p + "norm2b"] = vec(W, 1.0, 0.1), vec(W, 1.0, 0.1)
                w[p + "mlp.up"], w[p + "mlp.down"] = mat(la.ff, W), mat(W, la.ff)
        return w

    @classmethod
    def random_init(cls, cfg: SozanexArgs, device="cuda", dtype=torch.bfloat16, seed=1234):
        return cls(cfg, cls.random_weights(cfg, device, dtype, seed), device, dtype).eval()

    def weight_bytes(self, ignore_embeddings=False) -> int:
        skip = {"embed", "bigram"} if ignore_embeddings else set()
        return sum(b.numel() * b.element_size() for n, b in self.named_buffers() if n not in skip)

    # ------------------------------------------------------------------------------------------------ state
    def setup_caches(self, max_batch_size, max_seq_length, dtype=None, device=None, kv_cache_quantization=False):
        """Per-sequence state for `max_batch_size` slots, one set per layer run: a ring of keys and values as long as the window
        (attention), latents and rotated key parts of up to max_seq_length positions (latent attention); and the last token
        (the embedding's).  A sequence may grow past max_seq_length when nothing had to be cut to it.  Same call as the Llama's
        setup_caches."""
        if kv_cache_quantization:
            raise NotImplementedError("Sozanex keeps its keys, values and latents in the model's dtype")
        if self.states is not None and self.max_seq_length >= max_seq_length and self.max_batch_size >= max_batch_size:
            return
        cfg, dev, n = self.config, self.device, max_batch_size
        self.max_batch_size, self.max_seq_length = max_batch_size, max_seq_length
        self.run_state = []
        bounded = False
        for i in cfg.runs:
            la, rs = cfg.layers[i], _RunState()
            m = la.mixer
            bounded |= m.window > max_seq_length
            rows = min(m.window, max_seq_length)
            if la.type == "attention":
                rs.window = WindowKVCache(n, rows, 0, m.kv_heads * m.dim, m.kv_heads * m.vdim, self.dtype, dev)
            else:
                rs.latent = LatentKVCache(n, rows, m.kv_rank, m.rot_dim, self.dtype, dev)
            self.run_state.append(rs)
        if cfg.bigram:
            rs = _RunState()
            rs.last = LastTokenState(n, dev)
            self.run_state.append(rs)
        self.states = SequenceStates(n, max_seq_length if bounded else 1 << 30)
        for rs in self.run_state:
            for part in rs.parts():
                self.states.on_grow.append(part.grow)
        self.states.on_grow.append(lambda k: setattr(self, "max_batch_size", k))
        self._step = None

    def state_bytes_per_sequence(self) -> int:
        return sum(b.numel() * b.element_size() for rs in self.run_state for part in rs.parts() for b in part.buffers()) \
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
        LAST position [B][1][vocab] in fp32 (what generation samples from).  The Llama's forward call shape.  Rings and the last
        token move with the sequence: positions must continue where the slots stand (or restart at 0)."""
        assert self.states is not None, "Caches must be initialized first"
        B, T = idx.shape
        start = 0 if input_pos is None else int(input_pos[0])
        st = self.states
        segs = []
        for b in range(B):
            slot = st.slot_of(("batch", b))
            assert slot == b, "generation batches own slots 0 .. B-1: release other requests first"
            assert start == 0 or st.length[slot] == start, "a sequence cannot jump to another position"
            st.length[slot] = start
            segs.append((slot, idx[b]))
        logits = self.step_engine.step(segs, want="last")
        return logits.view(B, 1, -1)
