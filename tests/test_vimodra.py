"""Vimodra against the plain definition in ``vimodra_oracle.py``: mechanisms one by one, prompts in portions, decoding, windows, pools.

Every test runs on the CPU (the operators' PyTorch definitions: cache, state and scheduler logic) and, marked ``gpu``, through the
kernels in fp32 and in bf16.
"""
import json
import os
import subprocess
import sys

import pytest
import torch

import vimodra_oracle as O
from adaptivetrainingsystem_b200.config import VimodraConfig
from adaptivetrainingsystem_b200.inference import ContinuousBatcher, GenerationEngine, SamplingParams, SequencePool, TraceRunner
from adaptivetrainingsystem_b200.models import Vimodra, load_model
from adaptivetrainingsystem_b200.ops import delta as delta_ops
from adaptivetrainingsystem_b200.ops import dyt as dyt_ops
from adaptivetrainingsystem_b200.ops import latent as latent_ops
from layered_utils import EXACT, PLACES, TOL, close, gpu, position_errors, run_portions, tokens


def build(cfg, weights, device, dtype):
    return Vimodra.from_tensors(VimodraConfig.from_dict(cfg), lambda n: weights[n], list(weights), dtype, device)


def mixed_config(**kw):
    layers = [O.with_mlp(O.latent_spec(size=9), 88), O.with_mlp(O.delta_spec(), 40), O.latent_spec(heads=5, dim=8, rot_dim=16, vdim=8, kv_rank=24, q_rank=32, size=21),
              O.with_mlp(O.delta_spec(heads=6, kv_heads=2, dim=24, vdim=16, conv=5), 56)]
    return O.config(layers, **{"width": 72, "loop": (1, 3, 2), **kw})


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("device,dtype", PLACES)
def test_norm_residual_gelu_steps(device, dtype):
    g = torch.Generator().manual_seed(0)
    T, K, N = 11, 40, 72

    def rnd(*s):
        return torch.randn(*s, generator=g)
    a, w, bias, x = rnd(T, K).to(dtype), rnd(N, K).to(dtype) * 0.2, rnd(N), rnd(T, N) * 3
    c = dyt_ops.DytChain(rnd(N), rnd(N), 0.6, rnd(N), rnd(N), 1.7)
    y = a.double() @ w.double().T + bias.double()
    want_x = x.double() + O.dyt(y, c.w1.double(), c.b1.double(), c.a1)
    want_h = O.dyt(want_x, c.w2.double(), c.b2.double(), c.a2)
    want_u = O.gelu_tanh(y)
    dev = dyt_ops.DytChain(c.w1.to(device), c.b1.to(device), c.a1, c.w2.to(device), c.b2.to(device), c.a2)
    xd = x.to(device)
    h = dyt_ops.linear_residual(a.to(device), w.to(device), bias.to(device), xd, dev)
    u = dyt_ops.linear_gelu(a.to(device), w.to(device), bias.to(device))
    assert xd.dtype == torch.float32 and h.dtype == dtype
    assert float((xd.cpu() - want_x).abs().max()) < 2e-5          # the residual is fp32 in both forms
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    assert float((h.float().cpu() - want_h).abs().max()) < tol and float((u.float().cpu() - want_u).abs().max() / want_u.abs().max()) < tol
    ids = torch.tensor([0, 6, 3])
    table, add = rnd(7, N).to(dtype), rnd(N)
    xe, he = dyt_ops.embed_norm(ids.to(device), table.to(device), add.to(device), dev.w2, dev.b2, dev.a2)
    want = table[ids].float() + add
    assert torch.equal(xe.cpu(), want) and float((he.float().cpu() - O.dyt(want, c.w2, c.b2, c.a2)).abs().max()) < tol


def _one_layer(layer, **kw):
    cfg = O.config([layer], **kw)
    return cfg, O.random_weights(cfg, seed=3)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("spec", [dict(), dict(heads=1, dim=32, rot_dim=2, vdim=33, kv_rank=17, q_rank=9, size=1), dict(heads=4, dim=20, rot_dim=12, size=64),
                                  dict(heads=2, dim=64, rot_dim=64, vdim=64, kv_rank=128, q_rank=64, size=33),
                                  dict(heads=3, dim=128, rot_dim=24, vdim=128, kv_rank=56, q_rank=40, size=50),
                                  dict(heads=3, dim=32, rot_dim=32, vdim=24, kv_rank=128, q_rank=40, size=20),
                                  dict(heads=18, dim=64, rot_dim=64, vdim=64, kv_rank=256, q_rank=64, size=70)])
def test_latent_attention_alone(device, dtype, spec):
    cfg, W = _one_layer(O.latent_spec(**spec))
    ids = tokens(70)
    want, streams = O.forward(cfg, W, ids)
    m, got = build(cfg, W, device, dtype), []
    logits = m(torch.tensor([ids], device=device), collect=got)
    close(logits[0], want, dtype)
    close(got[0][0], streams[0], dtype)
    close(run_portions(m, ids, [1] * 30 + [7, 2, 1, 30]), want, dtype)


def plain_window_attention(q, kv, kr, gate, s, n_old):
    """One sequence: q [L, H, dim + rot] rotated, kv / kr of n_old + L rows."""
    L, H = q.shape[:2]
    rows = n_old + L
    out = torch.empty(L, H, s.vdim, dtype=q.dtype)
    for i in range(L):
        lo, hi = max(0, n_old + i - s.window + 1), n_old + i + 1
        for h in range(H):
            k = torch.cat([kv[lo:hi, h * s.dim:(h + 1) * s.dim], kr[lo:hi]], 1)
            p = torch.softmax(k @ q[i, h] * s.scale, 0)
            out[i, h] = p @ kv[lo:hi, s.v_col + h * s.vdim:s.v_col + (h + 1) * s.vdim]
    assert rows == kv.shape[0]
    return out.reshape(L, -1) * torch.sigmoid(gate)


@gpu
@pytest.mark.parametrize("dims", [(128, 64, 128), (64, 64, 64), (64, 32, 128), (128, 8, 64)])
@pytest.mark.parametrize("L,n_old,window", [(300, 0, 1), (300, 0, 97), (513, 100, 101), (256, 255, 256), (128, 0, 1 << 30), (129, 37, 128), (400, 60, 129),
                                            (17, 500, 501), (640, 0, 384), (257, 0, 127)])
def test_tensor_core_window_attention(dims, L, n_old, window):
    """Query tiles of 128 / 256 rows, key blocks of 128: windows at, below and above their sizes, context before the portion, tails;
    keys at distance window - 1 carry a large score, so that the window's edge shows."""
    dim, rot, vdim = dims
    s = latent_ops.LatentShape(2, dim, rot, vdim, 64, 32, window, 0.11, 1e-5)
    g = torch.Generator().manual_seed(L + window)
    B = 2
    q, kv = torch.randn(B, L, s.q_width, generator=g), torch.randn(B, n_old + L, s.kv_width, generator=g)
    ctx, gate = torch.randn(B, n_old + L, s.cwp, generator=g), torch.randn(B, L, s.o_pad, generator=g)
    for edge in (window - 1, window):      # just inside and just outside: query i = 1.2 x the key at that distance, for every seventh query
        for i in range(L):
            j = n_old + i - edge
            if i % 7 == (0 if edge == window else 3) and j >= 0:
                for h in range(2):
                    q[:, i, h * (dim + rot):h * (dim + rot) + dim] = 1.2 * kv[:, j, h * dim:(h + 1) * dim]
    q, kv, ctx, gate = (v.to(torch.bfloat16) for v in (q, kv, ctx, gate))
    assert latent_ops.window_tc_ok(q.cuda(), s, L)
    out = latent_ops.window_attention(q.cuda().view(B * L, -1), kv.cuda(), ctx.cuda(), gate.cuda().view(B * L, -1), s, n_old).float().cpu().view(B, L, -1)
    for b in range(B):
        want = plain_window_attention(q[b].double().view(L, 2, -1), kv[b].double(), ctx[b, :, s.rank:s.cw].double(), gate[b].double(), s, n_old)
        assert float((out[b] - want).abs().max()) < 3e-2


@gpu
@pytest.mark.parametrize("H,dim,rot,vdim,rank,R", [(16, 128, 64, 128, 512, 300), (20, 32, 32, 40, 128, 64), (5, 64, 128, 64, 384, 1000), (33, 96, 32, 8, 256, 65)])
def test_tensor_core_latent_decode(H, dim, rot, vdim, rank, R):
    """Sequences of unequal length on one ring size: shorter than a tile, at a tile's and a chunk's edge, full rings that have wrapped
    around; one row of every sequence stands out in the scores."""
    s = latent_ops.LatentShape(H, dim, rot, vdim, rank, 32, R, 0.09, 1e-5)
    g = torch.Generator().manual_seed(R)
    lens = [0, 1, 31, 62, 63, 64, R - 2, R - 1, R, 3 * R + 5]
    lens = [min(x, 3 * R + 5) for x in lens] * 2
    B = len(lens)
    ring = torch.randn(B, R, s.cwp, generator=g)
    q, gate = torch.randn(B, s.q_width, generator=g), torch.randn(B, s.o_pad, generator=g)
    uk, uv = torch.randn(H * dim, rank, generator=g) / rank ** 0.5, torch.randn(H * vdim, rank, generator=g) / rank ** 0.5
    for b, n in enumerate(lens):
        row = (b * 37) % min(n + 1, R)
        ring[b, row, :rank] = (q[b, :dim] @ uk[:dim]) * 2      # head 0 looks at this row
    ring, q, gate, uk, uv = (v.to(torch.bfloat16) for v in (ring, q, gate, uk, uv))
    f = 1.0 / (777.0 ** (torch.arange(0, rot, 2).double() / rot))
    ang = torch.arange(3 * R + 6).double()[:, None] * f
    cos, sin = ang.cos().float().cuda(), ang.sin().float().cuda()
    lengths = torch.tensor(lens, dtype=torch.int32, device="cuda")
    ukt = uk.view(H, dim, rank).transpose(1, 2).contiguous().cuda()
    uvt = torch.zeros(H, rank, latent_ops.pad8(vdim), dtype=torch.bfloat16)
    uvt[..., :vdim] = uv.view(H, vdim, rank).transpose(1, 2)
    assert latent_ops.decode_mma_ok(s, torch.bfloat16)
    args = (q.cuda(), ring.cuda(), uk.cuda(), uvt.cuda(), gate.cuda(), s, cos, sin, lengths)
    got = {"tensor cores": latent_ops.latent_decode(*args, ukt, uv.cuda()), "general": latent_ops.latent_decode(*args)}
    for b, n in enumerate(lens):
        c = ring[b, :min(n + 1, R)].double()
        qb = q[b, :H * (dim + rot)].double().view(H, dim + rot)
        u, v = qb[:, dim:dim + rot // 2], qb[:, dim + rot // 2:]
        a = n * f
        qr = torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()], -1)
        k = (c[:, :rank] @ uk.double().T).view(-1, H, dim)
        vals = (c[:, :rank] @ uv.double().T).view(-1, H, vdim)
        p = torch.softmax((torch.einsum("hd,nhd->hn", qb[:, :dim], k) + qr @ c[:, rank:s.cw].T) * s.scale, -1)
        want = torch.einsum("hn,nhv->hv", p, vals).reshape(-1) * torch.sigmoid(gate[b, :H * vdim].double())
        for name, o in got.items():
            assert float((o[b, :H * vdim].float().cpu() - want).abs().max()) < 4e-2, (name, b, n)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("spec", [dict(), dict(heads=3, kv_heads=3, dim=5, vdim=7, conv=1), dict(heads=4, kv_heads=1, dim=40, vdim=130, conv=2),
                                  dict(heads=2, kv_heads=1, dim=128, vdim=64, conv=4), dict(heads=4, kv_heads=2, dim=64, vdim=128, conv=2),
                                  dict(heads=2, kv_heads=2, dim=8, vdim=256, conv=3), dict(heads=1, kv_heads=1, dim=200, vdim=16, conv=6)])
def test_delta_rule_alone(device, dtype, spec):
    cfg, W = _one_layer(O.delta_spec(**spec))
    ids = tokens(70)
    want, streams = O.forward(cfg, W, ids)
    m, got = build(cfg, W, device, dtype), []
    logits = m(torch.tensor([ids], device=device), collect=got)
    close(logits[0], want, dtype)
    close(got[0][0], streams[0], dtype)
    close(run_portions(m, ids, [1] * 9 + [2, 3, 2, 1, 8, 9, 1, 17, 18]), want, dtype)


@pytest.mark.parametrize("device,dtype", EXACT)
def test_delta_state_and_tail_after_portions(device, dtype):
    """The carried state itself: portions and single tokens leave the state of the plain recurrence behind."""
    s = delta_ops.DeltaShape(4, 2, 24, 20, 3, 1e-5)
    g = torch.Generator().manual_seed(5)
    n, B = 37, 2
    proj = torch.randn(B, n, s.proj_width, generator=g)
    conv, rate, dt = torch.randn(s.channels, s.taps, generator=g) * 0.6, -torch.rand(4, generator=g), torch.randn(4, generator=g) - 2
    state, tail = torch.full((B, 4, 24, 20), 7.0, device=device), torch.full((B, 2, s.channels), 9.0, device=device)   # leftovers
    at, outs = 0, []
    for L in (2, 11, 1, 1, 16, 6):
        part = proj[:, at:at + L].contiguous().to(device)
        lengths = torch.full((B,), at, dtype=torch.int32, device=device) if L == 1 else None
        mixed, rlen, gb = delta_ops.delta_prep(part, s, conv.T.contiguous().to(device), rate.to(device), dt.to(device), tail, at, lengths)
        if L == 1:
            delta_ops.delta_step(mixed, rlen, gb, state, part.view(B, -1)[:, s.g_col:], torch.ones(20, device=device), s, lengths)
        else:
            outs.append(delta_ops.delta_scan(mixed, rlen, gb, state, s, L, fresh=at == 0).view(B, L, -1))
        at += L
    kd = 2 * 24
    for b in range(B):
        x = proj[b].double()
        mix = O.silu(O.short_conv(x[:, :s.channels], conv.double()))
        q, k, v = mix[:, :kd].view(n, 2, 24), mix[:, kd:2 * kd].view(n, 2, 24), mix[:, 2 * kd:].view(n, 4, 20)
        q = (q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * 24 ** -0.5).repeat_interleave(2, 1)
        k = (k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)).repeat_interleave(2, 1)
        beta = torch.sigmoid(x[:, s.b_col:s.b_col + 4])
        dec = torch.exp(rate.double() * torch.log1p(torch.exp(x[:, s.a_col:s.a_col + 4] + dt.double())))
        o, S = O.delta_recurrence(q, k, v, beta, dec)
        assert float((state[b].cpu() - S).abs().max()) < 2e-5
        assert torch.equal(tail[b].cpu(), proj[b, -2:, :s.channels])
        assert float((outs[1][b].cpu() - o[2:13].reshape(11, -1)).abs().max()) < 2e-5
        assert float((outs[-1][b].cpu() - o[-6:].reshape(6, -1)).abs().max()) < 2e-5


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("kw", [dict(), dict(loop=None), dict(loop=(0, 4, 3), width=65, vocab=101), dict(loop=(3, 4, 1), eps=1e-3)])
def test_whole_prompt_layer_by_layer(device, dtype, kw):
    cfg = mixed_config(**kw)
    W = O.random_weights(cfg, seed=2)
    ids = tokens(61, cfg["vocab"])
    want, streams = O.forward(cfg, W, ids)
    m, got = build(cfg, W, device, dtype), []
    close(m(torch.tensor([ids], device=device), collect=got)[0], want, dtype)
    assert len(got) == len(streams)
    for a, b in zip(got, streams):
        close(a[0], b, dtype)
    assert float(position_errors(O.forward(cfg, W, ids, mistake="no_gate")[0].float(), want).max()) > 3 * TOL[dtype]
    assert float(position_errors(O.forward(cfg, W, ids, mistake="no_decay")[0].float(), want).max()) > 3 * TOL[dtype]


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("sizes", [[2] * 30 + [1], [61], [13, 8, 2, 21, 1, 1, 15], [1] * 61, [40] + [1] * 21, [3] * 20 + [1]])
def test_portions_and_token_by_token(device, dtype, sizes):
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    ids = tokens(61)
    close(run_portions(build(cfg, W, device, dtype), ids, sizes), O.forward(cfg, W, ids)[0], dtype)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("start", [61, 1])
def test_window_edges_show(device, dtype, start):
    """A short window and moderate scores: the key at the window's edge carries weight, so a window that is one token off moves the
    logits of many positions; prompts (start = 61) and decoding after the first token (start = 1)."""
    cfg = O.config([O.latent_spec(heads=2, dim=16, rot_dim=4, vdim=16, kv_rank=24, q_rank=24, size=6, scale=0.1)], width=48)
    W = O.random_weights(cfg, seed=7)
    ids = tokens(61)
    want = O.forward(cfg, W, ids)[0]
    m = build(cfg, W, device, dtype)
    got = run_portions(m, ids, [start] + [1] * (61 - start))
    close(got, want, dtype)
    for mistake in ("window_wide", "window_narrow"):
        wrong = position_errors(O.forward(cfg, W, ids, mistake=mistake)[0].float(), want)
        assert int((wrong > 1.3 * TOL[dtype]).sum()) >= 10, (mistake, wrong.tolist())


@pytest.mark.parametrize("device,dtype", EXACT)
def test_far_tokens_reach_through_the_recurrence_only(device, dtype):
    """A change of the first token reaches the last position through the delta rule's state and not past the window of a model with
    attention only."""
    for layers, reaches in (([O.latent_spec(size=4)], False), ([O.latent_spec(size=4), O.delta_spec()], True)):
        cfg = O.config(layers)
        W = O.random_weights(cfg, seed=4)
        for k in W:
            if k.endswith("A_log"):
                W[k] = torch.full_like(W[k], -6.0)   # slow decay: the state remembers
        m, ids = build(cfg, W, device, dtype), tokens(50)
        other = [(ids[0] + 1) % 104] + ids[1:]
        d = [float((run_portions(m, a, [20, 20, 10])[-1] - run_portions(m, b, [50])[-1]).abs().max()) for a, b in ((ids, ids), (ids, other))]
        assert d[0] < 1e-4 and (d[1] > 1e-3 if reaches else d[1] < 1e-4), d


@pytest.mark.parametrize("device,dtype", PLACES)
def test_batch_of_equal_prompts_against_each_alone(device, dtype):
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    m = build(cfg, W, device, dtype)
    rows = [tokens(33, seed=s) for s in range(3)]
    cache = m.make_cache(3, 40)
    ids = torch.tensor(rows, device=device)
    parts = [m(ids[:, :19], cache=cache), m(ids[:, 19:20], cache=cache), m(ids[:, 20:33], cache=cache)]
    got = torch.cat(parts, 1)
    for b, row in enumerate(rows):
        close(got[b], O.forward(cfg, W, row)[0], dtype)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_long_decoding(device, dtype):
    cfg = O.config([O.latent_spec(size=16), O.delta_spec(conv=4)], width=40)
    W = O.random_weights(cfg, seed=6)
    ids = tokens(260)
    close(run_portions(build(cfg, W, device, dtype), ids, [3] + [1] * 257), O.forward(cfg, W, ids)[0], dtype)


# ------------------------------------------------------------------------------------------------ pools, scheduler, entry points
@pytest.mark.parametrize("device,dtype", PLACES)
def test_pool_rows_are_reused_and_do_not_disturb_each_other(device, dtype):
    """Unequal requests interleaved on two rows: portions of one while the other decodes, rows closed and opened again."""
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    m = build(cfg, W, device, dtype)
    pool = SequencePool(m, 2, 64)
    reqs = {n: tokens(n, seed=n) for n in (30, 17, 2, 45)}
    want = {n: O.forward(cfg, W, r)[0] for n, r in reqs.items()}
    got = {n: [] for n in reqs}

    def extend(n, slot, a, b, active):
        got[n].append(pool.extend(slot, reqs[n][a:b], logits_at=range(b - a), active=active).float().cpu())

    def decode(n, slot, a, b):
        for i in range(a, b):
            pool.last[slot] = reqs[n][i]
            got[n].append(pool.decode([slot])[slot:slot + 1].float().cpu())
    s30, s17 = pool.open(), pool.open()
    extend(30, s30, 0, 9, True)
    extend(17, s17, 0, 5, False)                 # half a prompt: must survive the other row's decode steps
    decode(30, s30, 9, 14)
    extend(17, s17, 5, 11, False)
    decode(30, s30, 14, 30)
    pool.close(s30)
    s45 = pool.open()
    assert s45 == s30 and pool.available == 0
    extend(45, s45, 0, 1, True)                  # a sequence that begins with one token, in a row that held another
    decode(45, s45, 1, 20)
    extend(17, s17, 11, 17, False)
    pool.close(s17)
    s2 = pool.open()
    extend(2, s2, 0, 2, False)
    decode(45, s45, 20, 45)
    for n in reqs:
        close(torch.cat(got[n]), want[n], dtype)


def greedy_oracle(cfg, W, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(O.forward(cfg, W, ids)[0][-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("device,dtype", EXACT)
def test_greedy_generation_through_engine_and_scheduler(device, dtype):
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    m = build(cfg, W, device, dtype)
    prompts = [tokens(n, seed=n) for n in (1, 6, 19, 2, 27)]
    want = [greedy_oracle(cfg, W, p, 10) for p in prompts]
    params = SamplingParams.from_mode("greedy", max_new_tokens=10)
    engine = GenerationEngine(m)
    for graph in ([False, True] if device == "cuda" else [False]):
        out = engine.generate(torch.tensor([prompts[2]], device=device), params, use_graph=graph)
        assert out["tokens"][0].tolist() == want[2]
    for chunk in (None, 1, 5):
        batcher = ContinuousBatcher(engine, max_batch=3, max_len=40, params=params, prefill_chunk=chunk)
        assert batcher.run(prompts) == want
        assert batcher.slots.available == 3


@gpu
def test_bf16_generation_prefers_the_oracle_tokens():
    """bf16 may break near ties: every generated token must be within rounding of the best one of the plain definition."""
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    m = build(cfg, W, "cuda", torch.bfloat16)
    prompts = [tokens(n, seed=n) for n in (4, 19, 11)]
    outs = ContinuousBatcher(GenerationEngine(m), max_batch=2, max_len=48, prefill_chunk=7).run(prompts, 16)
    for p, o in zip(prompts, outs):
        logits = O.forward(cfg, W, p + o)[0][len(p) - 1:-1]
        gap = logits.max(-1).values - logits.gather(1, torch.tensor(o)[:, None])[:, 0]
        assert len(o) == 16 and float(gap.max()) < 0.3, gap


@pytest.mark.parametrize("device,dtype", PLACES)
def test_trace_replay_from_a_model_folder(device, dtype, tmp_path):
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    O.save_model(str(tmp_path), cfg, W)
    runner = TraceRunner(load_model(str(tmp_path), dtype, device), 64)
    for rid, ids in (("a", tokens(40)), ("b", tokens(23, seed=9))):
        want, at = O.forward(cfg, W, ids)[0], 0
        for n in (7, 1, 2, 1, 1, 9, 1, 1):
            keep = sorted({0, n // 2, n - 1})
            rec = {"step": 0, "entries": [{"id": rid, "tokens": ids[at:at + n], "want": keep}], "end": [rid] if at + n == 23 else []}
            close(runner.step(rec), want[[at + k for k in keep]], dtype)
            assert runner.step({"step": 1, "entries": [], "end": []}) is None
            at += n
    assert runner.pool.available == 2


@gpu
def test_trace_program(tmp_path):
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    O.save_model(str(tmp_path / "m"), cfg, W)
    ids = tokens(12)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:10], "want": [3, 9]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": ids[10:11], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": ids[11:], "want": [0]}], "end": ["x"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "16"],
                       input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = O.forward(cfg, W, ids)[0]
    for step, at in ((0, [3, 9]), (2, [11])):
        raw = torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32).view(len(at), -1)
        close(raw, want[at], torch.float32)
    assert not (tmp_path / "1.f32").exists()


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=gpu)])
def test_command_line_continues_token_ids(device, tmp_path):
    import Chat
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    O.save_model(str(tmp_path), cfg, W)
    chat = Chat.ChatInterface(model_folder=str(tmp_path), device=device, mode="greedy")
    prompt = tokens(9)
    got, want = chat.continue_ids(prompt, 6), greedy_oracle(cfg, W, prompt, 6)
    assert len(got) == 6 and (device != "cpu" or got == want)
    with pytest.raises(SystemExit, match="quantize"):
        Chat.ChatInterface(model_folder=str(tmp_path), device=device, quantize="int4")


# ------------------------------------------------------------------------------------------------ configuration, folders
def test_configuration_round_trip_and_errors(tmp_path):
    d = mixed_config()
    cfg = VimodraConfig.from_dict(d)
    assert VimodraConfig.from_dict(cfg.to_dict()) == cfg
    assert [r for r in cfg.runs()] == O.layer_runs(d)
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][1]["mixer"].pop("heads"), lambda c: c["layers"][1]["mixer"].update(kv_heads=3),
                   lambda c: c["layers"][0]["mixer"].update(rot_dim=7), lambda c: c["loop"].update(stop=9)):
        bad = json.loads(json.dumps(d))
        change(bad)
        with pytest.raises(ValueError):
            VimodraConfig.from_dict(bad)
    W = O.random_weights(d)
    W.pop("l0.ls1")
    with pytest.raises(ValueError, match="missing"):
        build(d, W, "cpu", torch.float32)
    O.save_model(str(tmp_path), {**d, "architecture": "Nothing"}, O.random_weights(d))
    with pytest.raises(ValueError, match="unknown architecture"):
        load_model(str(tmp_path), torch.float32, "cpu")
