"""A plain, slow statement of the Sozanex design, one function per mechanism.  It shares no code with the package: tests
compare the package's kernels and step function against it.  Everything is computed in the dtype of the tensors it is given
(float64 by default: the weights' own rounding is the only one).  `w` maps checkpoint tensor names to tensors, `cfg` is the
checkpoint's config.json as a dict.
"""
import json
import math
import os
import struct

import torch

ROUND_BF16 = False      # rounding_noise() sets it: activations are rounded to bfloat16 where a bfloat16 run stores them


def _r(x):
    return x.to(torch.bfloat16).to(x.dtype) if ROUND_BF16 else x


def layer_norm(x, weight, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def bigram_row(previous, token, b):
    """Row of the bigram table for a token and the one in front of it (None: the sequence's first token)."""
    return b["buckets"] if previous is None else (previous * b["mul_prev"] + token * b["mul_cur"]) % b["buckets"]


def embedding(cfg, w, tokens):
    e = cfg["embedding"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * e["scale"]
    if e.get("bigram"):
        rows = [bigram_row(tokens[i - 1] if i else None, t, e["bigram"]) for i, t in enumerate(tokens)]
        x = x + w["bigram"][torch.tensor(rows)]
    return x


def stretched_frequencies(f, s):
    """Three bands by wavelength: short ones keep their frequency, long ones turn `factor` times slower, a blend between."""
    out = f.clone()
    for i, fi in enumerate(f.tolist()):
        turns = s["original"] * fi / (2.0 * math.pi)      # over the original context
        if turns < s["low"]:
            out[i] = fi / s["factor"]
        elif turns <= s["high"]:
            share = (turns - s["low"]) / (s["high"] - s["low"])
            out[i] = share * fi + (1.0 - share) * fi / s["factor"]
    return out


def ramped_frequencies(f, dims, base, s):
    """Slow pairs turn `factor` times slower, fast ones as before, with a linear ramp between the pairs that make `slow` and
    `fast` turns over the original context."""
    where = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), dims - 1)
    ramp = ((torch.arange(dims // 2, dtype=f.dtype) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp)


def frequencies(rot, dtype=torch.float64):
    """-> (frequency of every rotated pair [dims / 2], factor on cosine and sine)."""
    dims, base = rot["dims"], rot["base"]
    f = torch.tensor(base, dtype=dtype) ** (-2.0 * torch.arange(dims // 2, dtype=dtype) / dims)
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    if "high" in s:
        return stretched_frequencies(f, s), 1.0
    return ramped_frequencies(f, dims, base, s), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot, layout):
    """x [T][heads][dim]; the first rot["dims"] coordinates of every head turn by position * frequency; pairs are
    (i, i + dims/2) for layout "half", (2i, 2i + 1) for layout "interleaved"."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    half = dims // 2
    f, amp = frequencies(rot, x.dtype)
    ang = positions.to(x.dtype)[:, None] * f[None, :]
    c, s = (torch.cos(ang) * amp)[:, None, :], (torch.sin(ang) * amp)[:, None, :]
    out = x.clone()
    ia, ib = (slice(0, half), slice(half, dims)) if layout == "half" else (slice(0, dims, 2), slice(1, dims, 2))
    a, b = x[..., ia], x[..., ib]
    out[..., ia] = a * c - b * s
    out[..., ib] = b * c + a * s
    return out


def sink_softmax(q, k, v, scale, size=None, sink=None):
    """q [T][H][d], k [T][G][d], v [T][G][dv]; query i sees key j when 0 <= i - j < size (None: every j <= i); exp(sink[h])
    joins the denominator of head h."""
    T, H, _ = q.shape
    G, dv = k.shape[1], v.shape[-1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & ((i - j < size) if size else (j <= i))
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = ((q[:, hd] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        if sink is not None:
            s = torch.cat([s, sink[hd].expand(T, 1)], 1)
        out[:, hd] = torch.softmax(s, -1)[:, :T] @ v[:, g]
    return out


def attention(h, w, p, m, eps):
    """Grouped heads with biases, normed queries and keys, rotation, a sliding window.  Returns [T][H dv]."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d)
    v = _r(h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    q = rotate(rms_norm(q, w[p + "q.norm"], eps), pos, m.get("rot"), "half")
    k = rotate(rms_norm(k, w[p + "k.norm"], eps), pos, m.get("rot"), "half")
    return sink_softmax(_r(q), _r(k), v, m["scale"], (m.get("mask") or {}).get("size")).reshape(T, H * dv)


def latent_attention(h, w, p, m, eps):
    """Queries, keys and values through latents; one rotated key part for all heads; a sink; a gate on the concatenated
    heads.  Returns [T][H dv]."""
    T = h.shape[0]
    H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    cq = _r(rms_norm(_r(h @ w[p + "dq"].T), w[p + "dq.norm"], eps))
    q = _r(cq @ w[p + "uq"].T).view(T, H, dn + dr)
    ckv = _r(h @ w[p + "dkv"].T)
    c = _r(rms_norm(ckv[:, :R], w[p + "dkv.norm"], eps))
    kr = _r(rotate(ckv[:, R:].view(T, 1, dr), pos, m.get("rot"), "interleaved"))
    qr = _r(rotate(q[..., dn:], pos, m.get("rot"), "interleaved"))
    kn, v = _r(c @ w[p + "uk"].T).view(T, H, dn), _r(c @ w[p + "uv"].T).view(T, H, dv)
    q, k = torch.cat([q[..., :dn], qr], -1), torch.cat([kn, kr.expand(T, H, dr)], -1)
    o = sink_softmax(q, k, v, m["scale"], (m.get("mask") or {}).get("size"), w[p + "sink"]).reshape(T, H * dv)
    return o * torch.sigmoid(_r(h @ w[p + "g"].T))


def squared_relu(z):
    return torch.clamp(z, min=0.0) ** 2


def feed_forward(h, w, p):
    return _r(squared_relu(_r(h @ w[p + "up"].T))) @ w[p + "down"].T


def pass_input(x, x0, w):
    """What stands in front of a pass's first layer: one linear map of [residual; embedding output]."""
    return _r(torch.cat([x, x0], -1)) @ w["loop.in"].T


def layer(x, w, i, lay, eps):
    p, m = f"l{i}.", lay["mixer"]
    h = _r(layer_norm(x, w[p + "norm1"], eps))
    if lay["type"] == "attention":
        y = _r(attention(h, w, p + "mix.", m, eps)) @ w[p + "mix.o"].T + w[p + "mix.o.b"]
    else:
        y = _r(latent_attention(h, w, p + "mix.", m, eps)) @ w[p + "mix.o"].T
    x = x + layer_norm(y, w[p + "norm1b"], eps)
    if lay.get("mlp"):
        y = feed_forward(_r(layer_norm(x, w[p + "norm2"], eps)), w, p + "mlp.")
        x = x + layer_norm(y, w[p + "norm2b"], eps)
    return x


def order(cfg):
    """(layer, does a pass begin in front of it) of every layer run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    span = [(i, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return [(i, False) for i in range(lp["start"])] + span * lp["times"] + [(i, False) for i in range(lp["stop"], n)]


def forward(cfg, w, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T][vocab] of a whole sequence from position 0.  layers_out (a list) receives the residual after every layer run."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = x0 = embedding(cfg, w, list(tokens))
    for i, begins in order(cfg):
        if begins:
            x = pass_input(x, x0, w)
        x = layer(x, w, i, cfg["layers"][i], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return _r(layer_norm(x, w["final.norm"], eps)) @ w["head"].T


def rounding_noise(cfg, w, tokens, measure):
    """measure(exact logits, logits of the run that rounds to bfloat16 wherever a bfloat16 implementation does)."""
    global ROUND_BF16
    exact = forward(cfg, w, tokens)
    ROUND_BF16 = True
    try:
        rounded = forward(cfg, w, tokens)
    finally:
        ROUND_BF16 = False
    return measure(exact, rounded)


def greedy(cfg, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


# ------------------------------------------------------------------------------------------------ test models
def rotary(dims, base=500.0, ramp=None, bands=None):
    r = {"dims": dims, "base": base}
    if ramp:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), ramp))
    if bands:
        r["scaling"] = dict(zip(("factor", "original", "low", "high"), bands))
    return r


def attention_layer(heads=4, kv_heads=2, dim=12, vdim=8, scale=0.3, size=9, rot=8, base=300.0, bands=None, ff=40):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = rotary(rot, base, bands=bands)
    return {"type": "attention", "mixer": m, "mlp": dense(ff)}


def latent_layer(heads=3, dim=8, rot_dim=4, vdim=12, q_rank=10, kv_rank=14, scale=0.35, base=700.0, ramp=None, ff=40):
    return {"type": "latent_attention", "mlp": dense(ff),
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "rot": rotary(rot_dim, base, ramp)}}


def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def model_config(layers, width=32, vocab=61, eps=1e-5, scale=0.7, bigram=(37, 5, 11), loop=None):
    e = {"scale": scale}
    if bigram:
        e["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    cfg = {"architecture": "Sozanex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": e, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Every tensor the configuration names, seeded, sized so that each mechanism moves the logits."""
    gen = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(o, i, s=1.0):
        return torch.randn(o, i, generator=gen, dtype=torch.float32) * (s / math.sqrt(i))

    def vec(n, mean=0.0, s=1.0):
        return mean + s * torch.randn(n, generator=gen, dtype=torch.float32)

    w = {"embed": mat(V, W, 1.5 * math.sqrt(W)), "head": mat(V, W, 2.0), "final.norm": vec(W, 1.0, 0.2)}
    if cfg["embedding"].get("bigram"):
        w["bigram"] = mat(cfg["embedding"]["bigram"]["buckets"] + 1, W, 0.8 * math.sqrt(W))
    if cfg.get("loop"):
        w["loop.in"] = mat(W, 2 * W, 1.2)
    for i, lay in enumerate(cfg["layers"]):
        q, m = f"l{i}.mix.", lay["mixer"]
        w[f"l{i}.norm1"], w[f"l{i}.norm1b"] = vec(W, 1.0, 0.2), vec(W, 0.7, 0.2)
        H, dv = m["heads"], m["vdim"]
        if lay["type"] == "attention":
            G, d = m["kv_heads"], m["dim"]
            for s, n in (("q", H * d), ("k", G * d), ("v", G * dv)):
                w[q + s], w[q + s + ".b"] = mat(n, W), vec(n, 0.0, 0.4)
            w[q + "q.norm"], w[q + "k.norm"] = vec(d, 1.5, 0.4), vec(d, 1.5, 0.4)
            w[q + "o.b"] = vec(W, 0.0, 0.4)
        else:
            dn, dr, R, Rq = m["dim"], m["rot_dim"], m["kv_rank"], m["q_rank"]
            w[q + "dq"], w[q + "dq.norm"], w[q + "uq"] = mat(Rq, W), vec(Rq, 1.0, 0.2), mat(H * (dn + dr), Rq, 2.0)
            w[q + "dkv"], w[q + "dkv.norm"] = mat(R + dr, W, 1.5), vec(R, 1.0, 0.2)
            w[q + "uk"], w[q + "uv"] = mat(H * dn, R, 2.0), mat(H * dv, R)
            w[q + "sink"], w[q + "g"] = vec(H, 1.0, 1.0), mat(H * dv, W, 1.5)
        w[q + "o"] = mat(W, H * dv)
        f = lay.get("mlp")
        if f:
            w[f"l{i}.norm2"], w[f"l{i}.norm2b"] = vec(W, 1.0, 0.2), vec(W, 0.7, 0.2)
            w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"] = mat(f["ff"], W, 1.2), mat(W, f["ff"])
    return {k: v.to(dtype) for k, v in w.items()}


def write_checkpoint(folder, cfg, w):
    """config.json + model.safetensors (8-byte little-endian header length, JSON header, raw data) in `folder`."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    names = {torch.bfloat16: "BF16", torch.float32: "F32", torch.int32: "I32"}
    header, blobs, at = {}, [], 0
    for name, t in w.items():
        raw = t.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
