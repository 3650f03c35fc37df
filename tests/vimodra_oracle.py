"""Plain, slow definition of the Vimodra design, one function per mechanism, whole sequences only.

Nothing here is shared with the package: weights are a flat ``name -> tensor`` dictionary, every function takes a sequence
``[tokens, features]`` from position 0 and loops where the definition loops.  ``dtype`` (default float64) is the precision of
every operation.  The optional ``mistake`` argument of some functions plants one deliberate error, so that a test can show that its
inputs would reveal it.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def dyt(x, w, b, alpha):
    return torch.tanh(alpha * x) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def rotate_half(x, base):
    """x [tokens, .., dims], row t is position t; dimension i pairs with i + dims / 2."""
    n, dims = x.shape[0], x.shape[-1]
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = torch.arange(n, dtype=torch.float64)[:, None] * f
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    shape = [n] + [1] * (x.dim() - 2) + [half]
    c, s = c.view(shape), s.view(shape)
    u, v = x[..., :half], x[..., half:]
    return torch.cat([u * c - v * s, v * c + u * s], dim=-1)


def visible(n, size, mistake=None):
    """[query, key] boolean: key j of query i is seen when 0 <= i - j < size."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    if mistake == "window_wide":
        size += 1
    if mistake == "window_narrow":
        size -= 1
    return (d >= 0) & (d < size)


def latent_attention(W, p, m, h, eps, mistake=None):
    n, H = h.shape[0], m["heads"]
    dim, rd, vd, rank = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].T).view(n, H, dim + rd)
    ckv = h @ W[p + "dkv"].T
    c = rms(ckv[:, :rank], eps) * W[p + "dkv.norm"]
    kr = rotate_half(ckv[:, rank:], m["rot"]["base"])
    qu, qr = q[..., :dim], rotate_half(q[..., dim:], m["rot"]["base"])
    k = (c @ W[p + "uk"].T).view(n, H, dim)
    v = (c @ W[p + "uv"].T).view(n, H, vd)
    s = (torch.einsum("ihd,jhd->hij", qu, k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    s = s.masked_fill(~visible(n, m["mask"]["size"], mistake), float("-inf"))
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v).reshape(n, H * vd)
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


def delta_recurrence(q, k, v, beta, g, state=None):
    """q, k [tokens, heads, dim], v [tokens, heads, vdim], beta, g [tokens, heads] -> outputs [tokens, heads, vdim], final state."""
    n, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def delta_mixer(W, p, m, h, eps, mistake=None):
    n, H, KH, dim, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_conv(h @ W[p + "q"].T, W[p + "q.conv"])).view(n, KH, dim)
    k = silu(short_conv(h @ W[p + "k"].T, W[p + "k.conv"])).view(n, KH, dim)
    v = silu(short_conv(h @ W[p + "v"].T, W[p + "v.conv"])).view(n, H, vd)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * dim ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    src = torch.tensor([h_ // (H // KH) for h_ in range(H)])
    q, k = q[:, src], k[:, src]
    beta = torch.sigmoid(h @ W[p + "b"].T)
    a = h @ W[p + "a"].T + W[p + "dt_bias"]
    g = torch.exp(-torch.exp(W[p + "A_log"]) * torch.nn.functional.softplus(a, threshold=50))
    if mistake == "no_decay":
        g = torch.ones_like(g)
    o, _ = delta_recurrence(q, k, v, beta, g)
    o = rms(o, eps) * W[p + "norm"]
    o = o.reshape(n, H * vd) * silu(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def feed_forward(W, p, h):
    return gelu_tanh(h @ W[p + "up"].T + W[p + "up.b"]) @ W[p + "down"].T + W[p + "down.b"]


def layer_runs(cfg):
    """[(layer, pass or None)]: the order in which layers are run; the pass number is set on the first layer of a loop pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, None) for i in range(a)]
    for t in range(times):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg, weights, tokens, dtype=torch.float64, mistake=None):
    """-> (logits [tokens, vocab], [residual stream after every layer run])"""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return dyt(x, W[name], W[name + ".b"], W[name + ".alpha"])
    x = W["embed"][torch.as_tensor(tokens).long()]
    streams = []
    for i, t in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = x + W["loop.step"][t]
        mixer = latent_attention if L["type"] == "latent_attention" else delta_mixer
        y = mixer(W, p + "mix.", L["mixer"], norm(x, p + "norm1"), eps, mistake)
        x = x + norm(y, p + "norm1b") * W[p + "ls1"]
        if L["mlp"] is not None:
            x = x + norm(feed_forward(W, p + "mlp.", norm(x, p + "norm2")), p + "norm2b") * W[p + "ls2"]
        streams.append(x)
    return norm(x, "final.norm") @ W["head"].T, streams


# ----------------------------------------------------------------------------------------------------------------------------
# random models of the design
# ----------------------------------------------------------------------------------------------------------------------------
def latent_spec(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, q_rank=48, size=9, base=5000.0, scale=0.2):
    return {"type": "latent_attention", "mlp": None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "mask": {"size": size}, "rot": {"base": base, "dims": rot_dim}, "scale": scale}}


def delta_spec(heads=4, kv_heads=2, dim=16, vdim=24, conv=3):
    return {"type": "delta", "mlp": None, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def with_mlp(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def config(layers, width=72, vocab=104, loop=None, eps=1e-5):
    c = {"architecture": "Vimodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


def random_weights(cfg, seed=0, sharp=1.0):
    """bf16-representable float32 weights.  ``sharp`` scales the query projections, so that single keys stand out in the scores."""
    g = torch.Generator().manual_seed(seed)

    def mat(n, k, s=1.0):
        return torch.randn(n, k, generator=g) * (s / math.sqrt(k))

    def vec(n, mean=0.0, s=0.1):
        return mean + s * torch.randn(n, generator=g)
    D, V, W = cfg["width"], cfg["vocab"], {}
    W["embed"] = torch.randn(V, D, generator=g)
    W["head"] = mat(V, D, 1.5)

    def norm(name):
        W[name], W[name + ".b"], W[name + ".alpha"] = vec(D, 1.0, 0.3), vec(D, 0.0, 0.2), torch.tensor(0.7) + 0.2 * torch.rand((), generator=g)
    norm("final.norm")
    if cfg.get("loop"):
        W["loop.step"] = 0.5 * torch.randn(cfg["loop"]["times"], D, generator=g)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1"), norm(p + "norm1b")
        W[p + "ls1"] = vec(D, 0.8, 0.2)
        if L["type"] == "latent_attention":
            H = m["heads"]
            W[p + "mix.dq"], W[p + "mix.dq.norm"] = mat(m["q_rank"], D), vec(m["q_rank"], 1.0, 0.3)
            W[p + "mix.uq"] = mat(H * (m["dim"] + m["rot_dim"]), m["q_rank"], 2.0 * sharp)
            W[p + "mix.dkv"], W[p + "mix.dkv.norm"] = mat(m["kv_rank"] + m["rot_dim"], D, 1.5), vec(m["kv_rank"], 1.0, 0.3)
            W[p + "mix.uk"], W[p + "mix.uv"] = mat(H * m["dim"], m["kv_rank"], 2.0), mat(H * m["vdim"], m["kv_rank"], 2.0)
            W[p + "mix.g"], W[p + "mix.o"] = mat(H * m["vdim"], D, 2.0), mat(D, H * m["vdim"], 2.0)
        else:
            H, KH, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", KH * d), ("k", KH * d), ("v", H * vd)):
                W[p + "mix." + n], W[p + f"mix.{n}.conv"] = mat(rows, D, 2.0), torch.randn(rows, m["conv"], generator=g) * 0.6
            W[p + "mix.b"], W[p + "mix.a"] = mat(H, D, 2.0), mat(H, D, 1.0)
            W[p + "mix.A_log"], W[p + "mix.dt_bias"] = vec(H, -0.5, 1.0), vec(H, -2.0, 1.0)
            W[p + "mix.norm"], W[p + "mix.g"], W[p + "mix.o"] = vec(vd, 1.0, 0.3), mat(H * vd, D, 2.0), mat(D, H * vd, 2.0)
        if L["mlp"] is not None:
            norm(p + "norm2"), norm(p + "norm2b")
            W[p + "ls2"], ff = vec(D, 0.8, 0.2), L["mlp"]["ff"]
            W[p + "mlp.up"], W[p + "mlp.up.b"] = mat(ff, D, 1.5), vec(ff, 0.0, 0.3)
            W[p + "mlp.down"], W[p + "mlp.down.b"] = mat(D, ff, 1.5), vec(D, 0.0, 0.3)
    return {k: v.to(torch.bfloat16).float() for k, v in W.items()}


def save_model(folder, cfg, weights):
    """config.json + model.safetensors (bf16) as a user would have them."""
    import json
    import os
    import struct
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {}, [], 0
    for name, t in weights.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
