"""Serving throughput of a layer-listed design (``vimodra``, ``nemipel``) beside the closest other models of the framework (the dense
grouped-query decoder; for Nemipel also Vimodra) at equal width, depth, head count and feed-forward size, with random weights;
``bench.py --design NAME`` prints it.

``end_to_end`` times whole prompts and graph-replayed decode steps; ``kernels`` times the kernels of one layer of either model alone, with
L2 flushed before every launch, and puts each beside its roofline (the larger of FLOPs over the tensor or fp32 rate and bytes over the
copy bandwidth).  All times are CUDA events on the launching stream.
"""
from __future__ import annotations

import json
import os
import time
from typing import Any, Callable, Dict, List, Optional

import torch

# nominal sizes of a mid-size decoder; Vimodra: three latent-attention layers to one recurrent layer; Nemipel: lightning, attention and
# channel-wise delta layers in turn, the second attention layer on the first one's keys and values
SIZES: Dict[str, Dict[str, int]] = {
    "w2048": dict(width=2048, heads=16, kv_rank=512, q_rank=768, ff=8192),
    "w4096": dict(width=4096, heads=32, kv_rank=512, q_rank=1536, ff=16384),
}
LAYERS, VOCAB, WINDOW = 8, 32000, 1024
PEERS: Dict[str, List[str]] = {"vimodra": ["dense"], "nemipel": ["dense", "vimodra"]}   # models timed beside a design


def vimodra_config(size: str):
    from ..config import VimodraConfig
    z = SIZES[size]
    mlp = {"kind": "dense", "ff": z["ff"]}
    attn = {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": z["heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": z["kv_rank"], "q_rank": z["q_rank"],
                                                               "mask": {"size": WINDOW}, "rot": {"base": 10000.0, "dims": 64}, "scale": 192 ** -0.5}}
    rec = {"type": "delta", "mlp": mlp, "mixer": {"heads": z["heads"], "kv_heads": z["heads"] // 2, "dim": 128, "vdim": 128, "conv": 4}}
    return VimodraConfig.from_dict({"vocab": VOCAB, "width": z["width"], "norm": {"eps": 1e-5}, "layers": [rec if i % 4 == 3 else attn for i in range(LAYERS)]})


def gated_ff(size: str) -> int:
    """A gated feed-forward has three matrices: two thirds of the width for the same size."""
    return (2 * SIZES[size]["ff"] // 3 + 127) // 128 * 128


def nemipel_config(size: str):
    from ..config import NemipelConfig
    z = SIZES[size]
    H, mlp = z["heads"], {"kind": "dense", "ff": gated_ff(size)}
    light = {"type": "lightning", "mlp": mlp, "mixer": {"heads": H, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-1 - 8.0 * i / H) for i in range(H)]}}
    rec = {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": H, "kv_heads": H // 2, "dim": 128, "vdim": 128, "conv": 4}}

    def attn(**kw):
        return {"type": "attention", "mlp": mlp, "mixer": {"heads": H, "kv_heads": H // 4, "dim": 128, "vdim": 128, "rot": {"base": 10000.0, "dims": 64},
                                                            "scale": 128 ** -0.5, "softcap": 25.0, **kw}}
    layers = [light, attn(), rec, light, attn(kv_from=1), rec, light, attn()]
    assert len(layers) == LAYERS
    return NemipelConfig.from_dict({"vocab": VOCAB, "width": z["width"], "norm": {"eps": 1e-6}, "postln_alpha": 2.0, "logit_softcap": 20.0, "layers": layers})


def dense_config(size: str, seq: int):
    from ..config import ModelConfig
    z = SIZES[size]
    return ModelConfig(vocab_size=VOCAB, hidden_size=z["width"], num_layers=LAYERS, num_heads=z["heads"], num_kv_heads=z["heads"] // 4,
                       intermediate_size=gated_ff(size), seq_length=seq, tie_word_embeddings=False)


def build(design: str, size: str, seq: int):
    dev = torch.device("cuda", torch.cuda.current_device())
    if design != "dense":
        from ..models import Nemipel, Vimodra
        return Vimodra.random(vimodra_config(size), torch.bfloat16, dev) if design == "vimodra" else Nemipel.random(nemipel_config(size), torch.bfloat16, dev)
    from ..models import DeepSeekTransformer
    torch.manual_seed(0)
    with torch.device(dev):
        torch.set_default_dtype(torch.bfloat16)
        m = DeepSeekTransformer(dense_config(size, seq))
        torch.set_default_dtype(torch.float32)
    return m.eval()


def _events():
    return torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)


@torch.no_grad()
def end_to_end(design: str, size: str, prefill_batch: int = 8, prompt: int = 2048, decode_batches=(1, 64), new_tokens: int = 64, repeat: int = 3) -> Dict[str, Any]:
    from .. import ops
    from .engine import GenerationEngine, SamplingParams, sample_next
    model = build(design, size, prompt + new_tokens)
    eng = GenerationEngine(model)
    dev = next(model.parameters()).device
    g = torch.Generator().manual_seed(7)
    params = SamplingParams.from_mode("greedy")
    ids = torch.randint(0, VOCAB, (prefill_batch, prompt), generator=g).to(dev)
    times: List[float] = []
    for i in range(3 + repeat):
        cache = model.make_cache(prefill_batch, prompt)
        torch.cuda.synchronize()
        a, b = _events()
        a.record()
        eng.prefill(ids, cache)
        b.record()
        torch.cuda.synchronize()
        if i >= 3:
            times.append(a.elapsed_time(b))
        del cache
    ops.check_status()
    out: Dict[str, Any] = {"parameters": model.num_parameters(), "prefill_ms": min(times), "prefill_tokens_per_s": prefill_batch * prompt / min(times) * 1e3, "decode": {}}
    context = prompt // 2
    for B in decode_batches:
        rows = ids[:1, :context].expand(B, context).contiguous()
        cache = model.make_cache(B, context + new_tokens + 8)
        logits = eng.prefill(rows, cache)
        dec = eng.graph_decoder(cache)
        for _ in range(4):
            logits = dec.step(sample_next(logits, params))
        torch.cuda.synchronize()
        a, b = _events()
        a.record()
        for _ in range(new_tokens):
            logits = dec.step(sample_next(logits, params))
        b.record()
        torch.cuda.synchronize()
        ops.check_status()
        ms = a.elapsed_time(b) / new_tokens
        out["decode"][str(B)] = {"ms_per_step": ms, "tokens_per_s": B / ms * 1e3}
        del dec, cache
    del eng, model
    torch.cuda.empty_cache()
    return out


def peaks() -> Dict[str, Any]:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            d = json.load(f)
        if "hbm_gbs" in d and "bf16_tflops" in d:
            return {"bytes": d["hbm_gbs"] * 1e9, "flops": d["bf16_tflops"] * 1e12, "kind": "measured"}
    return {"bytes": 6.65e12, "flops": 1.59e15, "kind": "fallback"}


FP32_FLOPS = 148 * 128 * 2 * 1.965e9   # nominal: 128 FMA lanes per SM (the recurrence is fp32 by definition and has no tensor form here)


class _Timer:
    def __init__(self, dev, iters: int = 20):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
        self.iters, self.peak, self.rows = iters, peaks(), []

    def add(self, model: str, name: str, fn: Callable[[], Any], bytes_: float, flops: float = 0.0, fp32: float = 0.0) -> None:
        torch.cuda.synchronize()
        time.sleep(0.3)   # clocks that a heavy product before this one has pulled under the power cap recover
        for _ in range(3):
            fn()
        ts = []
        for _ in range(self.iters):
            self.flush.zero_()
            a, b = _events()
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        ts.sort()
        ms = ts[len(ts) // 2]
        roof = max(bytes_ / self.peak["bytes"], flops / self.peak["flops"], fp32 / FP32_FLOPS) * 1e3
        self.rows.append({"model": model, "kernel": name, "us": round(ms * 1e3, 1), "roofline_us": round(roof * 1e3, 2), "of_roofline": round(roof / ms, 3)})


def _bf(*shape):
    return torch.randn(*shape, device="cuda").to(torch.bfloat16)


def _gemm_cost(T, N, K, extra=0):
    return dict(bytes_=2.0 * (T * K + N * K + T * N) + extra, flops=2.0 * T * N * K)


@torch.no_grad()
def kernels(design: str, size: str, B: int = 8, L: int = 2048, decode_batch: int = 64) -> List[Dict[str, Any]]:
    """The kernels of one layer of every kind of ``design``, then those of the models beside it."""
    t = _Timer(torch.device("cuda", torch.cuda.current_device()))
    for name in [design] + PEERS[design]:
        {"vimodra": _vimodra_kernels, "nemipel": _nemipel_kernels, "dense": _dense_kernels}[name](t, size, B, L, decode_batch)
        torch.cuda.empty_cache()
    return t.rows


def _vimodra_kernels(t: _Timer, size: str, B: int, L: int, n: int) -> None:
    from .. import ops
    from ..ops import delta as D, dyt, latent as A
    m = build("vimodra", size, L)
    dev = next(m.parameters()).device
    z, W = SIZES[size], SIZES[size]["width"]
    att, rec, mlp = m.mixers[0], m.mixers[3], m.mlps[0]
    s, d = att.s, rec.s
    rope = att._rope[0]
    rope.ensure(L, dev)
    T = B * L
    H, ff = s.heads, z["ff"]

    bf, gemm_cost = _bf, _gemm_cost
    # ---- portions
    h, x = bf(T, W), torch.randn(T, W, device=dev)
    c1, c2 = m.chains[0]
    t.add("vimodra", "prefill gemm: q / kv latents + gate", lambda: ops.linear(h, att.w_in), **gemm_cost(T, s.proj_width, W))
    proj = ops.linear(h, att.w_in).view(B, L, -1)
    st = att.state(B, L, torch.bfloat16, dev)
    t.add("vimodra", "prefill latent_context", lambda: A.latent_context(proj, s, att.q_norm, att.kv_norm, rope.cos, rope.sin, st["ring"]), 2.0 * T * 2 * (s.q_rank + s.cw))
    cq, ctx, _ = A.latent_context(proj, s, att.q_norm, att.kv_norm, rope.cos, rope.sin, st["ring"])
    q = ops.linear(cq, att.w_uq)
    kv = ops.linear(ctx.view(-1, s.cwp)[:, :s.rank], att.w_ukv[:, :s.rank]).view(B, L, -1)
    t.add("vimodra", "prefill gemm: key / value expansion", lambda: ops.linear(ctx.view(-1, s.cwp)[:, :s.rank], att.w_ukv[:, :s.rank]), **gemm_cost(T, s.kv_width, s.rank))
    t.add("vimodra", "prefill latent_finish", lambda: A.latent_finish(q, ctx, st["ring"], s, rope.cos, rope.sin, 0, 0, L),
          2.0 * (2 * T * H * s.rot + 2 * B * min(L, WINDOW) * s.cw))
    gate = proj.view(T, -1)[:, s.g_col:]
    w = min(WINDOW, L)
    pairs = B * H * (w * (w + 1) / 2 + (L - w) * w)
    t.add("vimodra", "prefill window_attention", lambda: A.window_attention(q, kv, ctx, gate, s, 0), 2.0 * T * (s.q_width + s.kv_width + s.rot + 2 * s.o_pad),
          flops=2.0 * pairs * (s.dim + s.rot + s.vdim))
    a = A.window_attention(q, kv, ctx, gate, s, 0)
    t.add("vimodra", "prefill gemm + residual step: attention output", lambda: dyt.linear_residual(a, att.w_o, None, x, c1), **gemm_cost(T, W, s.o_pad, 8.0 * T * W))
    t.add("vimodra", "prefill gemm + gelu: up", lambda: mlp(h), **gemm_cost(T, ff, W))
    u = mlp(h)
    t.add("vimodra", "prefill gemm + residual step: down", lambda: dyt.linear_residual(u, mlp.w_down, mlp.b_down, x, c2), **gemm_cost(T, W, ff, 8.0 * T * W))
    dproj = ops.linear(h, rec.w_in).view(B, L, -1)
    ds = rec.state(B, L, torch.bfloat16, dev)
    t.add("vimodra", "prefill delta_prep", lambda: D.delta_prep(dproj, d, rec.conv, rec.neg_rate, rec.dt_bias, ds["tail"]), 2.0 * T * 2 * d.channels)
    mixed, rlen, gb = D.delta_prep(dproj, d, rec.conv, rec.neg_rate, rec.dt_bias, ds["tail"])
    t.add("vimodra", "prefill delta_scan", lambda: D.delta_scan(mixed, rlen, gb, ds["S"], d, L, True), 2.0 * T * (d.channels + d.heads * d.vdim),
          fp32=2.0 * T * d.heads * 3 * d.dim * d.vdim)
    o = D.delta_scan(mixed, rlen, gb, ds["S"], d, L, True)
    dg = dproj.view(T, -1)[:, d.g_col:]
    t.add("vimodra", "prefill delta_output", lambda: D.delta_output(o, dg, rec.norm, d), 2.0 * T * 3 * d.heads * d.vdim)
    del u, mixed, o, dproj, q, kv, a
    # ---- one token per sequence
    hd, xd = bf(n, W), torch.randn(n, W, device=dev)
    lengths = torch.full((n,), L - 1, dtype=torch.int32, device=dev)
    active = torch.ones(n, dtype=torch.int32, device=dev)
    sd = att.state(n, L, torch.bfloat16, dev)
    sd["ring"].normal_()
    pd = ops.linear(hd, att.w_in).view(n, 1, -1)
    t.add("vimodra", "decode latent_context", lambda: A.latent_context(pd, s, att.q_norm, att.kv_norm, rope.cos, rope.sin, sd["ring"], lengths=lengths, active=active),
          2.0 * n * 2 * (s.q_rank + s.cw))
    qd = bf(n, s.q_width)
    gd = pd.view(n, -1)[:, s.g_col:]
    t.add("vimodra", "decode latent attention (absorb + ring + expand)",
          lambda: att.attend_token(qd, sd["ring"], gd, lengths),
          2.0 * (n * w * s.cw + H * (s.dim + s.vdim) * s.rank), flops=2.0 * n * H * w * (s.cw + s.rank))
    t.add("vimodra", "decode gemm: q / kv latents + gate", lambda: ops.linear(hd, att.w_in), 2.0 * att.w_in.numel())
    ad = bf(n, s.o_pad)
    t.add("vimodra", "decode gemm + residual step: attention output", lambda: dyt.linear_residual(ad, att.w_o, None, xd, c1), 2.0 * att.w_o.numel())
    t.add("vimodra", "decode gemm + gelu: up", lambda: mlp(hd), 2.0 * mlp.w_up.numel())
    ud = bf(n, ff)
    t.add("vimodra", "decode gemm + residual step: down", lambda: dyt.linear_residual(ud, mlp.w_down, mlp.b_down, xd, c2), 2.0 * mlp.w_down.numel())
    dd, dpd = rec.state(n, L, torch.bfloat16, dev), ops.linear(hd, rec.w_in).view(n, 1, -1)
    t.add("vimodra", "decode delta_prep", lambda: D.delta_prep(dpd, d, rec.conv, rec.neg_rate, rec.dt_bias, dd["tail"], 0, lengths, active),
          2.0 * n * d.channels * (2 + 2 * (d.taps - 1)))
    mx, rl, gbd = D.delta_prep(dpd, d, rec.conv, rec.neg_rate, rec.dt_bias, dd["tail"], 0, lengths, active)
    t.add("vimodra", "decode delta_step", lambda: D.delta_step(mx, rl, gbd, dd["S"], dpd.view(n, -1)[:, d.g_col:], rec.norm, d, lengths, active),
          8.0 * n * d.heads * d.dim * d.vdim)
    ops.check_status()


def _nemipel_kernels(t: _Timer, size: str, B: int, L: int, n: int) -> None:
    from .. import ops
    from ..ops import delta as D, gqa as Q, lightning as N, postnorm as pn
    m = build("nemipel", size, L)
    dev = next(m.parameters()).device
    W, T = SIZES[size]["width"], B * L
    light, att, rec, mlp = m.mixers[0], m.mixers[1], m.mixers[2], m.mlps[0]
    ls, s, d, ff = light.s, att.s, rec.s, mlp.ff
    H, rope = s.heads, att._rope[0]
    rope.ensure(L + 1, dev)
    c1, c2 = m.steps[0]
    bf, gemm_cost, name = _bf, _gemm_cost, "nemipel"
    state = 4.0 * H * 128 * 128
    # ---- portions
    h, x = bf(T, W), torch.randn(T, W, device=dev)
    t.add(name, "prefill gemm + silu: lightning q, k, v, gate", lambda: pn.linear_silu(h, light.w_in, ls.g_col), **gemm_cost(T, ls.proj_width, W))
    proj, S = pn.linear_silu(h, light.w_in, ls.g_col), light.state(B, L, torch.bfloat16, dev)["S"]
    # products inside chunks of 128 tokens and with the state, everything once
    t.add(name, "prefill lightning attention", lambda: N.lightning_scan(proj, S, light.powers, ls, L, True), 2.0 * T * (ls.v_col + 2 * ls.o_pad),
          flops=2.0 * T * H * (64 * 256 + 2 * 128 * 128))
    o = N.lightning_scan(proj, S, light.powers, ls, L, True)
    t.add(name, "prefill norm_gate", lambda: pn.norm_gate(o, proj[:, ls.g_col:], light.norm, ls.eps, ls.o_pad), 2.0 * T * 3 * ls.o_pad)
    a = pn.norm_gate(o, proj[:, ls.g_col:], light.norm, ls.eps, ls.o_pad)
    t.add(name, "prefill gemm + post-norm step: attention output", lambda: pn.linear_postnorm(a, light.w_o, x, c1), **gemm_cost(T, W, ls.o_pad, 8.0 * T * W))
    part = torch.randn(1, T, W, device=dev)
    t.add(name, "prefill post-norm step alone", lambda: _fold_alone(pn, part, x, c1), 4.0 * T * W * 3 + 2.0 * T * W)
    del part
    t.add(name, "prefill gemm + swiglu: up", lambda: mlp(h), **gemm_cost(T, 2 * ff, W, -2.0 * T * ff))
    u = mlp(h)
    t.add(name, "prefill gemm + post-norm step: down", lambda: pn.linear_postnorm(u, mlp.w_down, x, c2), **gemm_cost(T, W, ff, 8.0 * T * W))
    del proj, o, a, u
    t.add(name, "prefill gemm: q, k, v, gate", lambda: ops.linear(h, att.w_in), **gemm_cost(T, s.proj_width, W))
    proj = ops.linear(h, att.w_in).view(B, L, -1)
    st = att.state(B, L, torch.bfloat16, dev)
    t.add(name, "prefill gqa_prepare (norms, rotation, cache)", lambda: Q.gqa_prepare(proj, s, att.q_norm, att.k_norm, rope.cos, rope.sin, st["k"], st["v"]),
          2.0 * T * 2 * (s.q_pad + s.k_pad + s.v_pad))
    q, gate = Q.gqa_prepare(proj, s, att.q_norm, att.k_norm, rope.cos, rope.sin, st["k"], st["v"]), proj.view(T, -1)[:, s.g_col:]
    t.add(name, "prefill attention (causal, capped)", lambda: Q.gqa_portion(q, st["k"], st["v"], gate, s, L, 0), 2.0 * T * (2 * s.q_pad + s.k_pad + s.v_pad),
          flops=2.0 * B * H * (L * (L + 1) / 2) * 2 * s.dim)
    del proj, q, gate, st
    t.add(name, "prefill gemm: delta q, k, v, low-rank inputs", lambda: ops.linear(h, rec.w_in), **gemm_cost(T, d.proj_width, W))
    proj = ops.linear(h, rec.w_in)
    low = proj[:, d.low_col:d.low_col + d.low_width]
    t.add(name, "prefill gemm: delta decays, gate", lambda: ops.linear(low, rec.w_low), **gemm_cost(T, d.g_col + d.o_pad, d.low_width / 2))
    wide, ds = ops.linear(low, rec.w_low), rec.state(B, L, torch.bfloat16, dev)
    t.add(name, "prefill delta_prep", lambda: D.delta_prep(proj.view(B, L, -1), d, rec.conv, None, None, ds["tail"]), 2.0 * T * 2 * d.channels)
    mixed, rlen, gb = D.delta_prep(proj.view(B, L, -1), d, rec.conv, None, None, ds["tail"])
    t.add(name, "prefill channel_delta_scan", lambda: D.channel_delta_scan(mixed, rlen, gb, wide, rec.neg_rate, rec.dt_bias, ds["S"], d, L, True),
          2.0 * T * (d.channels + d.heads * (d.dim + d.vdim)), fp32=2.0 * T * d.heads * 3 * d.dim * d.vdim)
    o = D.channel_delta_scan(mixed, rlen, gb, wide, rec.neg_rate, rec.dt_bias, ds["S"], d, L, True)
    t.add(name, "prefill delta_output", lambda: D.delta_output(o, wide[:, d.g_col:], rec.norm, d), 2.0 * T * 3 * d.heads * d.vdim)
    del proj, low, wide, mixed, o, h, x
    # ---- one token per sequence
    hd, xd = bf(n, W), torch.randn(n, W, device=dev)
    lengths, active = torch.full((n,), L - 1, dtype=torch.int32, device=dev), torch.ones(n, dtype=torch.int32, device=dev)
    t.add(name, "decode gemm + silu: lightning q, k, v, gate", lambda: pn.linear_silu(hd, light.w_in, ls.g_col), 2.0 * light.w_in.numel())
    pd, Sd = pn.linear_silu(hd, light.w_in, ls.g_col), light.state(n, L, torch.bfloat16, dev)["S"]
    t.add(name, "decode lightning_step", lambda: N.lightning_step(pd, Sd, light.decay, ls, lengths, active), 2 * n * state)
    od = N.lightning_step(pd, Sd, light.decay, ls, lengths, active)
    t.add(name, "decode norm_gate", lambda: pn.norm_gate(od, pd[:, ls.g_col:], light.norm, ls.eps, ls.o_pad), 2.0 * n * 3 * ls.o_pad)
    ad = bf(n, ls.o_pad)
    t.add(name, "decode gemm + post-norm step: attention output", lambda: pn.linear_postnorm(ad, light.w_o, xd, c1), 2.0 * light.w_o.numel())
    t.add(name, "decode gemm + swiglu: up", lambda: mlp(hd), 2.0 * mlp.w_gate_up.numel())
    ud = bf(n, ff)
    t.add(name, "decode gemm + post-norm step: down", lambda: pn.linear_postnorm(ud, mlp.w_down, xd, c2), 2.0 * mlp.w_down.numel())
    w = min(WINDOW, L)   # the cache length of the dense model's row
    sd = att.state(n, w + 8, torch.bfloat16, dev)
    sd["k"].normal_(), sd["v"].normal_()
    at = torch.full((n,), w - 1, dtype=torch.int32, device=dev)
    t.add(name, "decode gemm: q, k, v, gate", lambda: ops.linear(hd, att.w_in), 2.0 * att.w_in.numel())
    pa = ops.linear(hd, att.w_in).view(n, 1, -1)
    t.add(name, "decode gqa_prepare", lambda: Q.gqa_prepare(pa, s, att.q_norm, att.k_norm, rope.cos, rope.sin, sd["k"], sd["v"], 0, at, active),
          2.0 * n * 2 * (s.q_pad + s.k_pad + s.v_pad))
    qd, gd = bf(n, s.q_pad), pa.view(n, -1)[:, s.g_col:]
    t.add(name, "decode attention (capped, gated)", lambda: Q.gqa_decode(qd, sd["k"], sd["v"], gd, s, at), 2.0 * n * w * (s.k_pad + s.v_pad))
    t.add(name, "decode gemm: delta q, k, v, low-rank inputs", lambda: ops.linear(hd, rec.w_in), 2.0 * rec.w_in.numel())
    pr = ops.linear(hd, rec.w_in)
    t.add(name, "decode gemm: delta decays, gate", lambda: ops.linear(pr[:, d.low_col:d.low_col + d.low_width], rec.w_low), 2.0 * rec.w_low.numel())
    wd, dd = ops.linear(pr[:, d.low_col:d.low_col + d.low_width], rec.w_low), rec.state(n, L, torch.bfloat16, dev)
    t.add(name, "decode delta_prep", lambda: D.delta_prep(pr.view(n, 1, -1), d, rec.conv, None, None, dd["tail"], 0, lengths, active),
          2.0 * n * d.channels * (2 + 2 * (d.taps - 1)))
    mx, rl, gbd = D.delta_prep(pr.view(n, 1, -1), d, rec.conv, None, None, dd["tail"], 0, lengths, active)
    t.add(name, "decode delta_step", lambda: D.delta_step(mx, rl, gbd, dd["S"], wd[:, d.g_col:], rec.norm, d, lengths, active, wd, rec.neg_rate, rec.dt_bias),
          2 * n * state)
    lg = torch.randn(n, VOCAB, device=dev)
    t.add(name, "decode softcap of the logits", lambda: pn.softcap_(lg, 20.0, True), 8.0 * n * VOCAB)
    ops.check_status()


def _fold_alone(pn, part, x, c) -> None:
    """The fold launch of ``linear_postnorm`` without its product."""
    from .. import ops
    h = torch.empty(x.shape, dtype=torch.bfloat16, device=x.device)
    a = pn._PostNorm(part.data_ptr(), 1, x.numel(), x.data_ptr(), c.alpha, c.w.data_ptr(), 0, c.eps, h.data_ptr(), x.shape[0], x.shape[1], c.width)
    ops._lib.check(pn._fns().ats_fold_postnorm(pn.ctypes.byref(a), 0, ops._lib.stream_ptr(x.device)), "ats_fold_postnorm")


def _dense_kernels(t: _Timer, size: str, B: int, L: int, n: int) -> None:
    from .. import ops
    from ..ops import gemm as G
    bf, gemm_cost = _bf, _gemm_cost
    W, T, w = SIZES[size]["width"], B * L, min(WINDOW, L)
    dev = t.flush.device
    h, hd, ad = bf(T, W), bf(n, W), bf(n, W)
    p = build("dense", size, L)
    blk = p.layers[0]
    at = blk.self_attn
    I = blk.ffn.down_proj.shape[1]
    nkv, hd_ = at.n_kv, at.d
    p.rope.ensure(L, dev)
    t.add("dense", "prefill gemm: qkv", lambda: ops.linear(h, at.qkv_proj), **gemm_cost(T, at.qkv_proj.shape[0], W))
    qkv = ops.linear(h, at.qkv_proj).view(B, L, -1)
    t.add("dense", "prefill rope", lambda: ops.rope_packed(qkv, p.rope.cos, p.rope.sin, at.n_q, nkv, hd_), 2.0 * 2 * T * (at.n_q + nkv) * hd_)
    t.add("dense", "prefill rms_norm", lambda: ops.rms_norm(h, blk.input_norm.weight), 2.0 * 2 * T * W)
    t.add("dense", "prefill attention (causal)", lambda: ops.attention_packed(qkv, at.n_q, nkv, hd_), 2.0 * T * (at.n_q * 2 + 2 * nkv) * hd_,
          flops=2.0 * B * at.n_q * (L * (L + 1) / 2) * 2 * hd_)
    ao = bf(T, W)
    t.add("dense", "prefill gemm + residual: attention output", lambda: ops.linear(ao, at.o_proj, residual=h), **gemm_cost(T, W, W, 2.0 * T * W))
    t.add("dense", "prefill gemm + swiglu: up", lambda: G.gemm_nt_swiglu(h, blk.ffn.gate_up_proj), bytes_=2.0 * (T * W + 2 * I * W + T * I), flops=2.0 * T * 2 * I * W)
    ug = bf(T, I)
    t.add("dense", "prefill gemm + residual: down", lambda: ops.linear(ug, blk.ffn.down_proj, residual=h), **gemm_cost(T, W, I, 2.0 * T * W))
    kc, vc = bf(n, L, nkv, hd_), bf(n, L, nkv, hd_)
    lens = torch.full((n,), w - 1, dtype=torch.int32, device=dev)
    qd2 = bf(n, 1, at.qkv_proj.shape[0])
    kcw, vcw = kc[:, :w + 8].contiguous(), vc[:, :w + 8].contiguous()
    t.add("dense", "decode attention", lambda: ops.decode_attention(qd2, kcw, vcw, lens, at.n_q, nkv, hd_), 2.0 * 2 * n * w * nkv * hd_)
    t.add("dense", "decode gemm: qkv", lambda: ops.linear(hd, at.qkv_proj), 2.0 * at.qkv_proj.numel())
    t.add("dense", "decode gemm + residual + norm: attention output",
          lambda: ops.serving.out_proj_norm(ad[:, :W].contiguous(), at.o_proj, hd, blk.post_attn_norm.weight, 1e-6), 2.0 * at.o_proj.numel())
    t.add("dense", "decode gemm + swiglu: up", lambda: G.gemm_nt_swiglu(hd, blk.ffn.gate_up_proj), 2.0 * blk.ffn.gate_up_proj.numel())
    ud2 = bf(n, I)
    t.add("dense", "decode gemm + residual: down", lambda: ops.linear(ud2, blk.ffn.down_proj, residual=hd), 2.0 * blk.ffn.down_proj.numel())
    t.add("dense", "decode rms_norm", lambda: ops.rms_norm(hd, blk.input_norm.weight), 2.0 * 2 * n * W)
    ops.check_status()


def run(design: str = "vimodra", sizes: Optional[List[str]] = None, per_kernel: bool = True) -> Dict[str, Any]:
    res: Dict[str, Any] = {"metric": f"{design}_serving_tokens_per_sec", "unit": "tokens/s", "n_gpus": 1, "higher_is_better": True, "dtype": "bf16", "data": "synthetic",
                           "config": {"layers": LAYERS, "vocab": VOCAB, "window": WINDOW, "prefill": "8 x 2048 tokens", "decode": "after 1024 tokens, CUDA graph",
                                      "l2": "kernel timings flush L2 before every launch; whole steps exceed it"},
                           "roofline": peaks()["kind"], "sizes": {}}
    for size in sizes or list(SIZES):
        r: Dict[str, Any] = {d: end_to_end(d, size) for d in [design] + PEERS[design]}
        if per_kernel:
            r["kernels"] = kernels(design, size)
            torch.cuda.empty_cache()
        res["sizes"][size] = r
    first = res["sizes"][(sizes or list(SIZES))[0]]
    res["value"] = first[design]["prefill_tokens_per_s"]
    return res
