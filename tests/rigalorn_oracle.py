"""A plain, slow statement of the Rigalorn design, one function per mechanism, token by token where the design is a
recurrence.  It shares no code with the package: tests compare the package's kernels and step function against it.
Everything is computed in the dtype of the tensors it is given (float64 by default: the weights' own rounding is the only
one).  `w` maps checkpoint tensor names to tensors, `cfg` is the checkpoint's config.json as a dict.
"""
import math

import torch
import torch.nn.functional as F

ROUND_BF16 = False      # rounding_noise() sets it: activations are rounded to bfloat16 where a bfloat16 run stores them


def _r(x):
    return x.to(torch.bfloat16).to(x.dtype) if ROUND_BF16 else x


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(z):
    return z * torch.sigmoid(z)


def xielu(z, p, q):
    """Quadratic above zero, an exponential's excess over its tangent below, plus half the identity everywhere."""
    return torch.where(z > 0, F.softplus(p) * z * z, (0.5 + F.softplus(q)) * (torch.exp(z) - 1 - z)) + 0.5 * z


def frequencies(rot, dtype=torch.float64):
    """(frequency of every rotated pair [dims / 2], factor on cosine and sine).  With `scaling`, slow pairs turn `factor`
    times slower, fast ones as before, with a linear ramp between the pairs that make `slow` and `fast` turns over the
    original context."""
    dims, base = rot["dims"], rot["base"]
    i = torch.arange(dims // 2, dtype=dtype)
    f = torch.tensor(base, dtype=dtype) ** (-2.0 * i / dims)
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    where = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


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


def window_softmax(q, k, v, scale, size):
    """q [T][H][d], k [T][G][d], v [T][G][dv]; query i sees key j when 0 <= i - j < size (None: every j <= i)."""
    T, H, _ = q.shape
    G, dv = k.shape[1], v.shape[-1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & ((i - j < size) if size else (j <= i))
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = ((q[:, hd] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        out[:, hd] = torch.softmax(s, -1) @ v[:, g]
    return out


def _size(m):
    return (m.get("mask") or {}).get("size")


def mixed_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, w, p, m, v_first):
    """Grouped-head attention with projection biases under a sliding window; v_first: the first value-mixing layer's values
    (None: nothing is mixed in).  Returns ([T][H dv], this layer's values as cached)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rotate((h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d), pos, m.get("rot"), "half")
    k = rotate((h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d), pos, m.get("rot"), "half")
    v = _r((h @ w[p + "v"].T + w[p + "v.b"])).view(T, G, dv)
    if v_first is not None:
        v = _r(mixed_values(v, v_first.view(T, G, dv), w[p + "vmix"]))
    return window_softmax(_r(q), _r(k), v, m["scale"], _size(m)).reshape(T, H * dv), v


def latent_attention(h, w, p, m, eps):
    """Queries, keys and values through latents; one rotated key part for all heads.  Returns [T][H dv]."""
    T = h.shape[0]
    H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    cq = _r(rms_norm(_r(h @ w[p + "dq"].T), w[p + "dq.norm"], eps))
    q = _r(cq @ w[p + "uq"].T).view(T, H, dn + dr)
    ckv = _r(h @ w[p + "dkv"].T)
    c = _r(rms_norm(ckv[:, :R], w[p + "dkv.norm"], eps))
    kr = _r(rotate(ckv[:, R:].view(T, 1, dr), pos, m.get("rot"), "interleaved"))
    qr = rotate(q[..., dn:], pos, m.get("rot"), "interleaved")
    kn, v = _r(c @ w[p + "uk"].T).view(T, H, dn), _r(c @ w[p + "uv"].T).view(T, H, dv)
    q = torch.cat([q[..., :dn], _r(qr)], -1)
    k = torch.cat([kn, kr.expand(T, H, dr)], -1)
    return window_softmax(q, k, v, m["scale"], _size(m)).reshape(T, H * dv)


def causal_conv(x, kernel):
    """x [T][C], kernel [C][taps], the last tap on the current row, zeros in front of the start."""
    T, C = x.shape
    taps = kernel.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x], 0)
    return sum(pad[j:j + T] * kernel[:, j] for j in range(taps))


def delta_recurrence(q, k, v, g, beta):
    """Per head S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q; q, k [T][G][d], v [T][H][dv], g, beta [T][H]."""
    T, H, dv = v.shape
    G, d = q.shape[1], q.shape[2]
    o = torch.zeros(T, H, dv, dtype=v.dtype)
    for hd in range(H):
        gr = hd // (H // G)
        S = torch.zeros(d, dv, dtype=v.dtype)
        for t in range(T):
            S = g[t, hd] * S
            u = beta[t, hd] * (v[t, hd] - S.T @ k[t, gr])
            S = S + torch.outer(k[t, gr], u)
            o[t, hd] = S.T @ q[t, gr]
    return o


def delta_inputs(h, w, p, m):
    """-> unit queries (scaled) and keys [T][G][d], values [T][H][dv], decays and step sizes [T][H]."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (_r(silu(causal_conv(_r(h @ w[p + s].T), w[p + s + ".conv"]))) for s in "qkv")
    q = unit_vector(q.view(T, G, d)) * d ** -0.5
    k = unit_vector(k.view(T, G, d))
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * F.softplus(h @ w[p + "a"].T + w[p + "dt_bias"], threshold=1e9))
    return q, k, v.view(T, H, dv), g, beta


def delta(h, w, p, m, eps):
    """Gated delta rule.  Returns [T][H dv]."""
    T = h.shape[0]
    o = delta_recurrence(*delta_inputs(h, w, p, m))
    o = rms_norm(o, w[p + "norm"], eps)
    return o.reshape(T, -1) * silu(_r(h @ w[p + "g"].T))


def feed_forward(h, w, p):
    act = w[p + "act"]
    return _r(xielu(_r(h @ w[p + "up"].T), act[0], act[1])) @ w[p + "down"].T


def forward(cfg, w, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T][vocab] of a whole sequence from position 0.  layers_out (a list) receives the residual after every layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    v_first = None
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", lay["mixer"]
        h = _r(rms_norm(x, w[f"l{i}.norm1"], eps))
        if lay["type"] == "attention":
            mixes = m.get("v_mix", False)
            o, v = attention(h, w, p, m, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = v
        elif lay["type"] == "delta":
            o = delta(h, w, p, m, eps)
        else:
            o = latent_attention(h, w, p, m, eps)
        y = _r(o) @ w[p + "o"].T
        if lay.get("mlp"):
            y = y + feed_forward(h, w, f"l{i}.mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return _r(rms_norm(x, w["final.norm"], eps)) @ w["head"].T


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
def rotary(dims, base=500.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def attention_layer(heads=4, kv_heads=2, dim=12, vdim=8, scale=0.3, size=9, rot=8, base=300.0, scaling=None, v_mix=False, ff=40):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = rotary(rot, base, scaling)
    if v_mix:
        m["v_mix"] = True
    return {"type": "attention", "mixer": m, "mlp": dense(ff)}


def delta_layer(heads=4, kv_heads=2, dim=8, vdim=12, conv=3, ff=40):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": dense(ff)}


def latent_layer(heads=3, dim=8, rot_dim=4, vdim=12, q_rank=10, kv_rank=14, scale=0.35, size=11, base=700.0, ff=40):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": rotary(rot_dim, base)}
    if size:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m, "mlp": dense(ff)}


def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def model_config(layers, width=32, vocab=61, eps=1e-5, scale=0.7):
    return {"architecture": "Rigalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Every tensor the configuration names, seeded, sized so that each mechanism moves the logits."""
    gen = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(o, i, s=1.0):
        return torch.randn(o, i, generator=gen, dtype=torch.float32) * (s / math.sqrt(i))

    def vec(n, mean=0.0, s=1.0):
        n = n if isinstance(n, tuple) else (n,)
        return mean + s * torch.randn(*n, generator=gen, dtype=torch.float32)

    w = {"embed": vec((V, W), 0.0, 1.5), "head": mat(V, W, 2.0), "final.norm": vec(W, 1.0, 0.2)}
    for i, lay in enumerate(cfg["layers"]):
        q, m = f"l{i}.mix.", lay["mixer"]
        w[f"l{i}.norm1"] = vec(W, 1.0, 0.2)
        H = m["heads"]
        if lay["type"] == "attention":
            G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
            for s, n, f in (("q", H * d, 2.0), ("k", G * d, 2.0), ("v", G * dv, 1.0)):
                w[q + s], w[q + s + ".b"] = mat(n, W, f), vec(n, 0.0, 0.3)
            if m.get("v_mix"):
                w[q + "vmix"] = torch.tensor(0.3 + 0.1 * (i % 4))
        elif lay["type"] == "delta":
            G, d, dv, taps = m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for s, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
                w[q + s], w[q + s + ".conv"] = mat(n, W, 1.5), vec((n, taps), 0.3, 0.5)
            w[q + "b"], w[q + "a"], w[q + "g"] = mat(H, W, 1.5), mat(H, W, 1.0), mat(H * dv, W, 1.5)
            w[q + "A_log"], w[q + "dt_bias"], w[q + "norm"] = vec(H, -1.0, 1.0), vec(H, -1.0, 1.0), vec(dv, 1.0, 0.3)
        else:
            dn, dr, dv, R, Rq = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            w[q + "dq"], w[q + "dq.norm"], w[q + "uq"] = mat(Rq, W), vec(Rq, 1.0, 0.2), mat(H * (dn + dr), Rq, 2.0)
            w[q + "dkv"], w[q + "dkv.norm"] = mat(R + dr, W, 1.5), vec(R, 1.0, 0.2)
            w[q + "uk"], w[q + "uv"] = mat(H * dn, R, 2.0), mat(H * dv, R)
            dv = m["vdim"]
        w[q + "o"] = mat(W, H * dv)
        f = lay.get("mlp")
        if f:
            r = f"l{i}.mlp."
            w[r + "up"], w[r + "down"], w[r + "act"] = mat(f["ff"], W, 1.2), mat(W, f["ff"]), vec(2, 0.2, 0.5)
    return {k: v.to(dtype) for k, v in w.items()}


def write_checkpoint(folder, cfg, w):
    """config.json + model.safetensors (8-byte little-endian header length, JSON header, raw data) in `folder`."""
    import json
    import os
    import struct
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
