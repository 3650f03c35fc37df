"""Plain, slow definition of the Nemipel design, one function per mechanism, whole sequences only.

Nothing here is shared with the package: weights are a flat ``name -> tensor`` dictionary, every function takes a sequence
``[tokens, features]`` from position 0 and loops where the definition loops.  ``dtype`` (default float64) is the precision of
every operation.  The optional ``mistake`` argument plants one deliberate error, so that a test can show that its inputs would
reveal it.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def rotate_pairs(x, dims, base, mistake=None):
    """x [tokens, heads, dim], row t is position t; of the first ``dims`` dimensions, 2i and 2i + 1 turn by t * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        a = torch.arange(x.shape[0], dtype=torch.float64) * f
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        p, q = (i, i + dims // 2) if mistake == "half_rotation" else (2 * i, 2 * i + 1)
        u, v = x[..., p], x[..., q]
        out[..., p], out[..., q] = u * c - v * s, v * c + u * s
    return out


def attention_keys(W, p, m, h, eps, mistake=None):
    """-> rotated keys [tokens, kv_heads, dim] and values [tokens, kv_heads, vdim]."""
    n, G = h.shape[0], m["kv_heads"]
    k = h @ W[p + "k"].T
    if mistake == "head_norm":
        k = (rms(k.view(n, G, -1), eps).reshape(n, -1)) * W[p + "k.norm"]
    else:
        k = rms(k, eps) * W[p + "k.norm"]
    k = rotate_pairs(k.view(n, G, m["dim"]), m["rot"]["dims"], m["rot"]["base"], mistake)
    return k, (h @ W[p + "v"].T).view(n, G, m["vdim"])


def attention_values(q, k, v, scale, cap, mistake=None):
    """q [tokens, H, dim], k [tokens, G, dim], v [tokens, G, vdim] -> [tokens, H, vdim]; every token sees itself and all before it."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(n, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G) if mistake != "head_order" else h % G
        for i in range(n):
            first = 1 if mistake == "no_first" and i > 0 else 0
            s = (k[first:i + 1, g] @ q[i, h]) * scale
            if cap is not None and mistake != "no_cap":
                s = softcap(s, cap)
            out[i, h] = torch.softmax(s, 0) @ v[first:i + 1, g]
    return out


def attention_mixer(W, p, m, h, eps, shared, mistake=None):
    """``shared``: keys and values of the layer named by ``kv_from``, or ``None``.  -> (output, keys and values)."""
    n, H = h.shape[0], m["heads"]
    k, v = shared if shared is not None else attention_keys(W, p, m, h, eps, mistake)
    q = rms(h @ W[p + "q"].T, eps) * W[p + "q.norm"]
    q = rotate_pairs(q.view(n, H, m["dim"]), m["rot"]["dims"], m["rot"]["base"], mistake)
    o = attention_values(q, k, v, m["scale"], m["softcap"], mistake)
    if mistake != "no_gate":
        o = o * torch.sigmoid(h @ W[p + "g"].T)[..., None]
    return o.reshape(n, -1) @ W[p + "o"].T, (k, v)


def lightning_recurrence(q, k, v, decay, state=None):
    """q, k [tokens, heads, dim], v [tokens, heads, vdim], decay [heads] -> outputs [tokens, heads, vdim], final state."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def lightning_mixer(W, p, m, h, eps, mistake=None):
    n, H = h.shape[0], m["heads"]
    q, k = silu(h @ W[p + "q"].T).view(n, H, -1), silu(h @ W[p + "k"].T).view(n, H, -1)
    v = silu(h @ W[p + "v"].T).view(n, H, -1)
    decay = torch.tensor(m["decay"], dtype=h.dtype)
    if mistake == "no_decay":
        decay = torch.ones_like(decay)
    o, _ = lightning_recurrence(q, k, v, decay)
    if mistake == "head_norm":
        o = rms(o, eps).reshape(n, -1) * W[p + "norm"]
    else:
        o = rms(o.reshape(n, -1), eps) * W[p + "norm"]
    if mistake != "no_gate":
        o = o * torch.sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def short_conv(x, w):
    """Causal per-channel convolution over time; the last column of ``w`` [channels, taps] weighs the current token."""
    n, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(n):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                y[t] = y[t] + w[:, j] * x[src]
    return y


def channel_recurrence(q, k, v, beta, g, state=None):
    """q, k, g [tokens, heads, dim], v [tokens, heads, vdim], beta [tokens, heads] -> outputs [tokens, heads, vdim], final state."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(q.shape[0]):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def channel_decay(a, A_log, dt_bias, heads):
    """a [tokens, heads * dim] -> decays [tokens, heads, dim]; one rate per head."""
    z = a + dt_bias
    sp = torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0)))).view(a.shape[0], heads, -1)
    return torch.exp(-torch.exp(A_log)[:, None] * sp)


def channel_delta_mixer(W, p, m, h, eps, mistake=None):
    n, H, KH, dim, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(name):
        return silu(short_conv(h @ W[p + name].T, W[p + name + ".conv"]))
    q, k, v = branch("q").view(n, KH, dim), branch("k").view(n, KH, dim), branch("v").view(n, H, vd)
    src = torch.tensor([h_ // (H // KH) for h_ in range(H)])
    if mistake == "head_order":
        src = torch.tensor([h_ % KH for h_ in range(H)])
    q, k = (unit(q) * dim ** -0.5)[:, src], unit(k)[:, src]
    beta = torch.sigmoid(h @ W[p + "b"].T)
    g = channel_decay((h @ W[p + "a1"].T) @ W[p + "a2"].T, W[p + "A_log"], W[p + "dt_bias"], H)
    if mistake == "no_decay":
        g = torch.ones_like(g)
    if mistake == "head_decay":
        g = g.mean(-1, keepdim=True).expand_as(g)
    o, _ = channel_recurrence(q, k, v, beta, g)
    o = rms(o, eps) * W[p + "norm"]
    gate = (h @ W[p + "g1"].T) @ W[p + "g2"].T
    if mistake != "no_gate":
        o = o * torch.sigmoid(gate).view(n, H, vd)
    return o.reshape(n, -1) @ W[p + "o"].T


def feed_forward(W, p, h):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def forward(cfg, weights, tokens, dtype=torch.float64, mistake=None):
    """-> (logits [tokens, vocab], [residual stream after every layer])"""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    if mistake == "no_alpha":
        alpha = 1.0
    x = W["embed"][torch.as_tensor(tokens).long()]
    streams, caches = [], {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        if L["type"] == "lightning":
            y = lightning_mixer(W, p + "mix.", m, x, eps, mistake)
        elif L["type"] == "channel_delta":
            y = channel_delta_mixer(W, p + "mix.", m, x, eps, mistake)
        else:
            y, caches[i] = attention_mixer(W, p + "mix.", m, x, eps, caches[m["kv_from"]] if "kv_from" in m else None, mistake)
        x = rms(alpha * x + y, eps) * W[p + "norm1"]
        if L["mlp"] is not None:
            x = rms(alpha * x + feed_forward(W, p + "mlp.", x), eps) * W[p + "norm2"]
        streams.append(x)
    return softcap((rms(x, eps) * W["final.norm"]) @ W["head"].T, cfg["logit_softcap"]), streams


# ----------------------------------------------------------------------------------------------------------------------------
# random models of the design
# ----------------------------------------------------------------------------------------------------------------------------
def lightning_spec(heads=3, dim=16, vdim=24, decay=None):
    decay = decay or [1.0 - 0.5 / (1.7 ** i) for i in range(heads)]
    return {"type": "lightning", "mlp": None, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def attention_spec(heads=4, kv_heads=2, dim=16, vdim=24, dims=8, base=5000.0, scale=0.3, cap=7.0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dims}, "scale": scale, "softcap": cap}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": None, "mixer": m}


def channel_delta_spec(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, a_rank=10, g_rank=6):
    """``a_rank`` / ``g_rank``: inner widths of the decay and gate projections (read from the tensors' shapes, not from the layer)."""
    return {"type": "channel_delta", "mlp": None, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "ranks": (a_rank, g_rank)}


def with_mlp(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def config(layers, width=72, vocab=104, eps=1e-3, alpha=1.7, cap=11.0):
    return {"architecture": "Nemipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "logit_softcap": cap, "layers": layers}


def random_weights(cfg, seed=0):
    """bf16-representable float32 weights."""
    g = torch.Generator().manual_seed(seed)

    def mat(n, k, s=1.0):
        return torch.randn(n, k, generator=g) * (s / math.sqrt(k))

    def vec(n, mean=0.0, s=0.1):
        return mean + s * torch.randn(n, generator=g)
    D, V, W = cfg["width"], cfg["vocab"], {}
    W["embed"], W["head"], W["final.norm"] = torch.randn(V, D, generator=g), mat(V, D, 3.0), vec(D, 1.0, 0.3)
    for i, L in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", L["mixer"], f"l{i}.mix."
        W[p + "norm1"] = vec(D, 1.0, 0.3)
        H, d, vd = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "lightning":
            W[q + "q"], W[q + "k"], W[q + "v"] = mat(H * d, D, 1.5), mat(H * d, D, 1.5), mat(H * vd, D, 1.5)
            W[q + "g"], W[q + "norm"], W[q + "o"] = mat(H * vd, D, 2.0), vec(H * vd, 1.0, 0.3), mat(D, H * vd, 3.0)
        elif L["type"] == "attention":
            G = m["kv_heads"]
            W[q + "q"], W[q + "q.norm"] = mat(H * d, D, 1.5), vec(H * d, 1.5, 0.3)
            if "kv_from" not in m:
                W[q + "k"], W[q + "k.norm"], W[q + "v"] = mat(G * d, D, 1.5), vec(G * d, 1.5, 0.3), mat(G * vd, D, 2.0)
            W[q + "g"], W[q + "o"] = mat(H, D, 2.0), mat(D, H * vd, 3.0)
        else:
            KH, (ra, rg) = m["kv_heads"], L["ranks"]
            for n, rows in (("q", KH * d), ("k", KH * d), ("v", H * vd)):
                W[q + n], W[q + n + ".conv"] = mat(rows, D, 2.0), torch.randn(rows, m["conv"], generator=g) * 0.6
            W[q + "b"], W[q + "a1"], W[q + "a2"] = mat(H, D, 2.0), mat(ra, D, 1.0), mat(H * d, ra, 1.0)
            W[q + "A_log"], W[q + "dt_bias"] = vec(H, -0.5, 1.0), vec(H * d, -2.0, 1.0)
            W[q + "norm"], W[q + "g1"], W[q + "g2"], W[q + "o"] = vec(vd, 1.0, 0.3), mat(rg, D, 1.5), mat(H * vd, rg, 1.5), mat(D, H * vd, 3.0)
        if L["mlp"] is not None:
            ff = L["mlp"]["ff"]
            W[p + "norm2"] = vec(D, 1.0, 0.3)
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = mat(ff, D, 1.5), mat(ff, D, 1.5), mat(D, ff, 2.0)
    return {k: v.to(torch.bfloat16).float() for k, v in W.items()}


def save_model(folder, cfg, weights):
    """config.json + model.safetensors (bf16) as a user would have them."""
    import json
    import os
    import struct
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump({**cfg, "layers": [{k: v for k, v in L.items() if k != "ranks"} for L in cfg["layers"]]}, f)
    head, blobs, at = {}, [], 0
    for name, t in weights.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
