"""Nemipel against the plain definition in ``nemipel_oracle.py``: mechanisms one by one, prompts in portions, decoding, shared caches, pools.

Every test runs on the CPU (the operators' PyTorch definitions: cache, state and scheduler logic) and, marked ``gpu``, through the
kernels in fp32 and in bf16.
"""
import json
import os
import subprocess
import sys

import pytest
import torch

import nemipel_oracle as O
from adaptivetrainingsystem_b200.config import NemipelConfig
from adaptivetrainingsystem_b200.inference import ContinuousBatcher, GenerationEngine, SamplingParams, SequencePool, TraceRunner
from adaptivetrainingsystem_b200.models import Nemipel, load_model
from adaptivetrainingsystem_b200.ops import delta as delta_ops
from adaptivetrainingsystem_b200.ops import gqa as gqa_ops
from adaptivetrainingsystem_b200.ops import lightning as lightning_ops
from adaptivetrainingsystem_b200.ops import postnorm as pn
from layered_utils import EXACT, PLACES, TOL, close, gpu, position_errors, run_portions, tokens

GPU_PLACES = PLACES[1:]
ALONE, WHOLE = 0.3, 0.6   # of the shared tolerance: one layer, and the mixed model (whose weight of the residual keeps roundings from growing)


def build(cfg, weights, device, dtype):
    return Nemipel.from_tensors(NemipelConfig.from_dict(cfg), lambda n: weights[n], list(weights), dtype, device)


def mixed_config(**kw):
    """Every kind of layer, with and without a feed-forward, two layers that share the first attention layer's keys and values."""
    layers = [O.lightning_spec(), O.with_mlp(O.attention_spec(), 88), O.with_mlp(O.channel_delta_spec(), 40), O.attention_spec(heads=6, kv_from=1),
              O.with_mlp(O.lightning_spec(heads=2, dim=24, vdim=8), 56), O.channel_delta_spec(heads=6, kv_heads=2, dim=24, vdim=16, conv=5),
              O.with_mlp(O.attention_spec(heads=5, kv_heads=5, dim=12, vdim=8, dims=12, cap=50.0), 32), O.attention_spec(heads=2, dims=8, cap=3.0, kv_from=1)]
    return O.config(layers, **{"alpha": 4.0, **kw})


def one_layer(layer, seed=3, **kw):
    cfg = O.config([layer], **kw)
    return cfg, O.random_weights(cfg, seed=seed)


def worst(a, b):
    """Largest difference over the largest value."""
    return float((a.double().cpu() - b.double()).abs().max() / b.double().abs().max())


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("T,K,width", [(11, 40, 69), (3, 2048, 72), (300, 64, 1000), (5, 24, 4100), (2, 16, 8200)])
def test_post_norm_residual_step(device, dtype, T, K, width):
    g = torch.Generator().manual_seed(0)
    N = (width + 7) // 8 * 8
    a, w, x = torch.randn(T, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) * 0.2).to(dtype), torch.randn(T, N, generator=g) * 3
    nw, nw2 = torch.randn(N, generator=g), torch.randn(N, generator=g)
    for t in (w, nw, nw2):
        t[width:] = 0
    x[:, width:] = 0
    want = O.rms((2.5 * x.double() + a.double() @ w.double().T)[:, :width], 1e-3) * nw.double()[:width]
    for second in (None, nw2):
        xd = x.to(device).clone()
        c = pn.PostNorm(2.5, nw.to(device), 1e-3, width, None if second is None else second.to(device))
        h = pn.linear_postnorm(a.to(device), w.to(device), xd, c)
        want_h = want if second is None else O.rms(want, 1e-3) * second.double()[:width]
        assert xd.dtype == torch.float32 and h.dtype == dtype
        assert float((xd.cpu()[:, :width] - want).abs().max()) < 4e-5      # the residual is fp32 in both forms
        assert float((h.float().cpu()[:, :width] - want_h).abs().max()) < (4e-5 if dtype == torch.float32 else 4e-2)
        assert not xd[:, width:].any() and not h[:, width:].any()


@pytest.mark.parametrize("device,dtype", PLACES)
def test_row_steps(device, dtype):
    g = torch.Generator().manual_seed(1)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for T, K, N, act in ((9, 40, 72, 48), (4, 2048, 264, 264), (5, 16, 24, 0)):
        a, w = torch.randn(T, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) * K ** -0.5).to(dtype)
        want = a.double() @ w.double().T
        want[:, :act] = O.silu(want[:, :act])
        assert worst(pn.linear_silu(a.to(device), w.to(device), act).float(), want) < tol
    for rows, n, pad in ((7, 70, 72), (3, 2048, 2048), (2, 5000, 5000), (3, 9000, 9000)):
        o, z, w = torch.randn(rows, pad + 8, generator=g).to(dtype), torch.randn(rows, pad, generator=g).to(dtype), torch.randn(n, generator=g)
        out = pn.norm_gate(o.to(device)[:, :pad], z.to(device), w.to(device), 1e-2, pad)
        assert worst(out[:, :n].float(), O.rms(o[:, :n].double(), 1e-2) * w.double() * torch.sigmoid(z[:, :n].double())) < tol
        assert not out[:, n:].any()
    z = torch.cat([torch.linspace(-90, 90, 397), torch.tensor([0.0, 1e-4, -1e-4])])
    for fast in (False, True):
        assert float((pn.softcap_(z.to(device).clone(), 13.0, fast).cpu() - O.softcap(z.double(), 13.0)).abs().max()) < 1e-5
    table = torch.randn(7, 72, generator=g).to(dtype)
    x, h = pn.embed_rows(torch.tensor([0, 6, 3], device=device), table.to(device))
    assert torch.equal(x.cpu(), table[[0, 6, 3]].float()) and torch.equal(h.cpu(), table[[0, 6, 3]])


ATTENTION_SPECS = [dict(), dict(heads=3, kv_heads=1, dim=10, vdim=7, dims=2), dict(heads=5, kv_heads=5, dim=24, vdim=40, dims=24, cap=60.0),
                   dict(heads=4, kv_heads=1, dim=64, vdim=64, dims=32, scale=0.15), dict(heads=16, kv_heads=2, dim=128, vdim=128, dims=64, scale=0.1, cap=4.0),
                   dict(heads=2, kv_heads=2, dim=128, vdim=72, dims=6, scale=0.1, cap=45.0), dict(heads=18, kv_heads=2, dim=40, vdim=16, dims=40, cap=2.0),
                   dict(heads=2, kv_heads=1, dim=160, vdim=200, dims=100, scale=0.1), dict(heads=4, kv_heads=2, cap=None)]


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("spec", ATTENTION_SPECS)
def test_attention_alone(device, dtype, spec):
    cfg, W = one_layer(O.attention_spec(**spec))
    ids = tokens(70)
    want, streams = O.forward(cfg, W, ids)
    m, got = build(cfg, W, device, dtype), []
    close(m(torch.tensor([ids], device=device), collect=got)[0], want, dtype, ALONE)
    close(got[0][0], streams[0], dtype, ALONE)
    close(run_portions(m, ids, [1] * 30 + [7, 2, 1, 30]), want, dtype, ALONE)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_attention_mistakes_would_show(device, dtype):
    """Rotation layout, norm over all heads, capped scores, key head of a query head, gate, the first token: each error moves the logits of
    this model beyond the tolerance."""
    spec = O.attention_spec(heads=6, kv_heads=3, dim=16, vdim=16, dims=16, base=50.0, scale=0.9, cap=2.5)
    cfg, W = one_layer(spec, alpha=0.5)
    ids = tokens(40)
    want = O.forward(cfg, W, ids)[0]
    close(build(cfg, W, device, dtype)(torch.tensor([ids], device=device))[0], want, dtype, ALONE)
    for mistake in ("half_rotation", "head_norm", "no_cap", "head_order", "no_gate", "no_first", "no_alpha"):
        assert float(position_errors(O.forward(cfg, W, ids, mistake=mistake)[0].float(), want).max()) > TOL[dtype], mistake


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,G,dim,vdim,cap", [(2, 1, 64, 64, 9.0), (4, 2, 128, 128, 30.0), (3, 3, 96, 80, 20.0), (2, 2, 72, 128, 70.0), (8, 1, 64, 64, 0.0), (2, 1, 18, 11, 12.0)])
@pytest.mark.parametrize("pos0,L", [(0, 300), (129, 17), (255, 2), (100, 157), (384, 129)])
def test_far_keys_in_portions_and_decoding(device, dtype, H, G, dim, vdim, cap, pos0, L):
    """Every query looks at one key that stands out among hundreds -- its own position, the first token, rows at the edges of key blocks and of
    the portion -- and is compared with the plain definition; the same keys for single queries at every cache length near an edge."""
    if device == "cpu" and (dim > 64 or L > 200):
        pytest.skip("covered by the smaller cases")
    s = gqa_ops.GqaShape(H, G, dim, vdim, 0, 0.5, cap, 1e-5)
    g = torch.Generator().manual_seed(pos0 + L)
    n, max_len = pos0 + L, pos0 + L + 9
    k, v = torch.full((2, max_len, s.k_pad), 3.0), torch.full((2, max_len, s.v_pad), 5.0)        # rows beyond the sequence hold leftovers
    k[:, :n, :G * dim], v[:, :n, :G * vdim] = torch.randn(2, n, G * dim, generator=g), torch.randn(2, n, G * vdim, generator=g)
    q, gate = torch.zeros(2, L, s.q_pad), torch.randn(2, L, H, generator=g)
    spots = [0, 1, 127, 128, 255, 256, pos0 - 1, pos0, pos0 + 1, n - 1]
    for i in range(L):
        for h in range(H):
            j = spots[(i + 3 * h) % len(spots)]
            j = j if 0 <= j <= pos0 + i else pos0 + i
            q[:, i, h * dim:(h + 1) * dim] = k[:, j, (h // (H // G)) * dim:][:, :dim] * (16.0 / dim)
    q, k, v, gate = (t.to(dtype) for t in (q, k, v, gate))
    want = []
    for b in range(2):
        full = torch.zeros(n, H, dim).double()
        full[pos0:] = q[b, :, :H * dim].double().view(L, H, dim)
        o = O.attention_values(full, k[b, :n, :G * dim].double().view(n, G, dim), v[b, :n, :G * vdim].double().view(n, G, vdim), 0.5, cap or None)[pos0:]
        want.append((o * torch.sigmoid(gate[b].double())[..., None]).reshape(L, -1))
    kd, vd, qd, gd = k.to(device), v.to(device), q.to(device).view(2 * L, -1), gate.to(device).view(2 * L, -1)
    tol = 1e-5 if dtype == torch.float32 else 1.5e-2
    out = gqa_ops.gqa_portion(qd, kd, vd, gd, s, L, pos0).view(2, L, -1)
    for b in range(2):
        assert worst(out[b, :, :H * vdim].float(), want[b]) < tol
    one = gqa_ops.gqa_portion(qd[L:], kd[1:], vd[1:], gd[L:], s, L, pos0)                        # a one-row view of the cache
    assert worst(one[:, :H * vdim].float(), want[1]) < tol
    for i in sorted({0, 1, L // 2, L - 2, L - 1}):
        lengths = torch.full((2,), pos0 + i, dtype=torch.int32, device=device)
        o = gqa_ops.gqa_decode(qd.view(2, L, -1)[:, i], kd, vd, gd.view(2, L, -1)[:, i], s, lengths)
        for b in range(2):
            assert worst(o[b, :H * vdim].float(), want[b][i]) < tol


@pytest.mark.parametrize("device,dtype", PLACES)
def test_prepare_norms_rotates_and_appends(device, dtype):
    for H, G, dim, vdim, rot in ((4, 2, 16, 24, 8), (3, 1, 10, 7, 10), (2, 2, 40, 8, 2)):
        s = gqa_ops.GqaShape(H, G, dim, vdim, rot, 1.0, 0.0, 1e-2)
        g = torch.Generator().manual_seed(dim)
        n, B, max_len = 13, 2, 20
        proj = torch.randn(B, n, s.proj_width, generator=g).to(dtype)
        qw, kw = torch.randn(H * dim, generator=g), torch.randn(G * dim, generator=g)
        ang = torch.arange(max_len + 1).double()[:, None] * 70.0 ** (-torch.arange(0, rot, 2).double() / rot)
        cos, sin = ang.cos().float().to(device), ang.sin().float().to(device)
        k, v = torch.zeros(B, max_len, s.k_pad, dtype=dtype, device=device), torch.zeros(B, max_len, s.v_pad, dtype=dtype, device=device)
        args = (s, qw.to(device), kw.to(device), cos, sin, k, v)
        q = [gqa_ops.gqa_prepare(proj[:, :5].contiguous().to(device), *args, pos0=0).view(B, 5, -1)]
        lengths, active = torch.tensor([5, 5], dtype=torch.int32, device=device), torch.tensor([1, 0], dtype=torch.int32, device=device)
        last = gqa_ops.gqa_prepare(proj[:, 5:6].contiguous().to(device), *args, lengths=lengths, active=active)
        q.append(last.view(B, 1, -1))
        assert not k[1, 5:].any() and not v[1, 5:].any()          # a row that sits out keeps its cache
        q.append(gqa_ops.gqa_prepare(proj[:, 6:].contiguous().to(device), *args, pos0=6).view(B, n - 6, -1))
        q, tol = torch.cat(q, 1).float().cpu(), 2e-5 if dtype == torch.float32 else 1e-2
        for b in range(B):
            x = proj[b].double()
            qn = (O.rms(x[:, :H * dim], 1e-2) * qw.double()).view(n, H, dim)
            kn = (O.rms(x[:, s.k_col:s.k_col + G * dim], 1e-2) * kw.double()).view(n, G, dim)
            assert worst(q[b, :, :H * dim], O.rotate_pairs(qn, rot, 70.0).reshape(n, -1)) < tol
            rows = [i for i in range(n) if (b, i) != (1, 5)]
            assert worst(k[b, rows, :G * dim].float(), O.rotate_pairs(kn, rot, 70.0).reshape(n, -1)[rows]) < tol
            assert torch.equal(v[b, rows, :G * vdim].cpu(), proj[b, rows, s.v_col:s.v_col + G * vdim])


@pytest.mark.parametrize("device,dtype", GPU_PLACES)
@pytest.mark.parametrize("dim,rot", [(16, 8), (10, 4)])
def test_prepare_long_and_short_portions_agree(device, dtype, dim, rot):
    """Many tokens and a handful of tokens are distributed over threads differently."""
    s = gqa_ops.GqaShape(4, 2, dim, 24, rot, 1.0, 0.0, 1e-3)
    n, g = 700, torch.Generator().manual_seed(1)
    proj = torch.randn(2, n, s.proj_width, generator=g).to(dtype).to(device)
    ang = torch.arange(n + 1).double()[:, None] * 50.0 ** (-torch.arange(0, rot, 2).double() / rot)
    consts = (s, torch.rand(4 * dim, generator=g).to(device), torch.rand(2 * dim, generator=g).to(device), ang.cos().float().to(device), ang.sin().float().to(device))
    results = []
    for step in (n, 100):
        k, v = torch.zeros(2, n, s.k_pad, dtype=dtype, device=device), torch.zeros(2, n, s.v_pad, dtype=dtype, device=device)
        q = [gqa_ops.gqa_prepare(proj[:, i:i + step].contiguous(), *consts, k, v, pos0=i).view(2, step, -1) for i in range(0, n, step)]
        results.append((torch.cat(q, 1).float(), k.float(), v.float()))
    for x, y in zip(*results):
        assert float((x - y).abs().max()) < (1e-5 if dtype == torch.float32 else 4e-2)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("spec", [dict(), dict(heads=5, dim=7, vdim=9), dict(heads=2, dim=64, vdim=64), dict(heads=1, dim=128, vdim=200, decay=[1.0]),
                                  dict(heads=3, dim=40, vdim=72, decay=[0.0, 0.3, 0.9999]), dict(heads=2, dim=200, vdim=16)])
def test_lightning_alone(device, dtype, spec):
    cfg, W = one_layer(O.lightning_spec(**spec))
    ids = tokens(150)
    want, streams = O.forward(cfg, W, ids)
    m, got = build(cfg, W, device, dtype), []
    close(m(torch.tensor([ids], device=device), collect=got)[0], want, dtype, ALONE)
    close(got[0][0], streams[0], dtype, ALONE)
    close(run_portions(m, ids, [1] * 9 + [2, 3, 2, 1, 33, 40, 60]), want, dtype, ALONE)
    if spec.get("heads", 3) > 1:
        assert float(position_errors(O.forward(cfg, W, ids, mistake="head_norm")[0].float(), want).max()) > TOL[dtype]


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,dim,vdim", [(3, 64, 64), (2, 128, 136), (4, 24, 40), (2, 12, 10)])
def test_lightning_chunks_and_state(device, dtype, H, dim, vdim):
    """Portions at, below and above the chunk of the tensor-core kernel from a state that is not zero; values that stand out at chunk edges;
    decays from 0 to 1; the state that is left behind."""
    s = lightning_ops.LightningShape(H, dim, vdim, tuple([1.0, 0.97, 0.2, 0.0][:H]), 1e-5)
    g = torch.Generator().manual_seed(dim)
    powers, decay = lightning_ops.decay_powers(s, device), torch.tensor(s.decay, dtype=torch.float64)
    sizes = (45, 1, 127, 128, 129, 2, 300) if device != "cpu" else (45, 1, 31)
    n, B = sum(sizes), 2
    proj = torch.randn(B, n, s.proj_width, generator=g) * 0.5
    for t in (0, 44, 45, 46, 172, 173, 300, 301, 429, 430, 431, n - 1):
        if t < n:
            proj[:, t, s.v_col:s.g_col] *= 40
    proj = proj.to(dtype)
    state = torch.full((B, H, dim, vdim), 7.0, device=device)   # leftovers
    at, outs = 0, []
    for L in sizes:
        part = proj[:, at:at + L].reshape(B * L, -1).contiguous().to(device)
        if L == 1:
            lengths = torch.full((B,), at, dtype=torch.int32, device=device)
            keep = state.clone()
            lightning_ops.lightning_step(part, state, powers[:, 1].contiguous(), s, lengths, torch.tensor([0, 0], dtype=torch.int32, device=device))
            assert torch.equal(keep, state)                      # rows that sit out
            o = lightning_ops.lightning_step(part, state, powers[:, 1].contiguous(), s, lengths)
        else:
            o = lightning_ops.lightning_scan(part, state, powers, s, L, fresh=at == 0)
        outs.append(o.view(B, L, -1)[..., :H * vdim].float().cpu())
        at += L
    got, tol = torch.cat(outs, 1), 1e-5 if dtype == torch.float32 else 6e-3
    for b in range(B):
        x = proj[b].double()
        q, k, v = x[:, :H * dim].view(n, H, dim), x[:, s.k_col:s.k_col + H * dim].view(n, H, dim), x[:, s.v_col:s.v_col + H * vdim].view(n, H, vdim)
        o, S = O.lightning_recurrence(q, k, v, decay)
        o = o.reshape(n, H, vdim)
        for h in range(H):
            assert worst(got[b].view(n, H, vdim)[:, h], o[:, h]) < tol
            # the state is carried in 32 bits whatever the element type (the decayed operands of the chunked form have 16 bits)
            assert worst(state[b, h], S[h]) < (5e-6 if dtype == torch.float32 else 3e-5)


CHANNEL_SPECS = [dict(), dict(heads=3, kv_heads=3, dim=5, vdim=7, conv=1, a_rank=3, g_rank=17), dict(heads=4, kv_heads=1, dim=40, vdim=130, conv=2, a_rank=1, g_rank=1),
                 dict(heads=2, kv_heads=1, dim=128, vdim=64, conv=4), dict(heads=4, kv_heads=2, dim=64, vdim=128, conv=2, a_rank=32, g_rank=40),
                 dict(heads=2, kv_heads=2, dim=8, vdim=256, conv=3), dict(heads=1, kv_heads=1, dim=200, vdim=16, conv=6)]


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("spec", CHANNEL_SPECS)
def test_channel_delta_alone(device, dtype, spec):
    cfg, W = one_layer(O.channel_delta_spec(**spec))
    ids = tokens(70)
    want, streams = O.forward(cfg, W, ids)
    m, got = build(cfg, W, device, dtype), []
    close(m(torch.tensor([ids], device=device), collect=got)[0], want, dtype, ALONE)
    close(got[0][0], streams[0], dtype, ALONE)
    close(run_portions(m, ids, [1] * 9 + [2, 3, 2, 1, 8, 9, 1, 17, 18]), want, dtype, ALONE)


@pytest.mark.parametrize("device,dtype", EXACT)
@pytest.mark.parametrize("H,KH,dim,vdim", [(4, 2, 24, 20), (2, 1, 72, 16), (2, 2, 130, 9)])
def test_channel_delta_state_and_tail_after_portions(device, dtype, H, KH, dim, vdim):
    """The carried state itself; decays from 1 down to an underflow within one token, different in every channel."""
    s = delta_ops.ChannelDeltaShape(H, KH, dim, vdim, 3, 1e-5, 6, 5)
    g = torch.Generator().manual_seed(5)
    n, B = 37, 2
    proj, wide = torch.randn(B, n, s.proj_width, generator=g), torch.randn(B, n, s.g_col + s.o_pad, generator=g) * 2
    conv, rate = torch.randn(s.channels, 3, generator=g) * 0.6, -torch.rand(H, generator=g) * 3
    dt = torch.linspace(-12, 60, H * dim)[torch.randperm(H * dim, generator=g)]
    state, tail = torch.full((B, H, dim, vdim), 7.0, device=device), torch.full((B, 2, s.channels), 9.0, device=device)   # leftovers
    at, outs = 0, []
    for L in (2, 11, 1, 1, 16, 6):
        part, w = proj[:, at:at + L].contiguous().to(device), wide[:, at:at + L].reshape(B * L, -1).contiguous().to(device)
        lengths = torch.full((B,), at, dtype=torch.int32, device=device) if L == 1 else None
        mixed, rlen, gb = delta_ops.delta_prep(part, s, conv.T.contiguous().to(device), None, None, tail, at, lengths)
        rates, bias = rate.to(device), dt.to(device)
        if L == 1:
            delta_ops.delta_step(mixed, rlen, gb, state, w[:, s.g_col:], torch.ones(vdim, device=device), s, lengths, None, w, rates, bias)
        else:
            outs.append(delta_ops.channel_delta_scan(mixed, rlen, gb, w, rates, bias, state, s, L, at == 0).view(B, L, -1))
        at += L
    kd = KH * dim
    for b in range(B):
        x = proj[b].double()
        mix = O.silu(O.short_conv(x[:, :s.channels], conv.double()))
        q, k, v = mix[:, :kd].view(n, KH, dim), mix[:, kd:2 * kd].view(n, KH, dim), mix[:, 2 * kd:].view(n, H, vdim)
        q, k = (O.unit(q) * dim ** -0.5).repeat_interleave(H // KH, 1), O.unit(k).repeat_interleave(H // KH, 1)
        beta = torch.sigmoid(x[:, s.b_col:s.b_col + H])
        dec = O.channel_decay(wide[b, :, :H * dim].double(), torch.log(-rate.double()), dt.double(), H)
        assert float(dec.min()) < 1e-30 and float(dec.max()) > 0.999
        o, S = O.channel_recurrence(q, k, v, beta, dec)
        assert float((state[b].cpu() - S).abs().max()) < 2e-5
        assert torch.equal(tail[b].cpu(), proj[b, -2:, :s.channels])
        assert float((outs[1][b].cpu() - o[2:13].reshape(11, -1)).abs().max()) < 2e-5
        assert float((outs[-1][b].cpu() - o[-6:].reshape(6, -1)).abs().max()) < 2e-5


@pytest.mark.parametrize("device,dtype", PLACES)
def test_recurrence_mistakes_would_show(device, dtype):
    for spec, mistakes in ((O.channel_delta_spec(heads=6, kv_heads=3), ("no_decay", "head_decay", "no_gate", "head_order")),
                           (O.lightning_spec(heads=4), ("no_decay", "no_gate", "head_norm"))):
        cfg, W = one_layer(spec, alpha=0.3)
        if spec["type"] == "channel_delta":
            W["l0.mix.dt_bias"] = (W["l0.mix.dt_bias"] * 3).to(torch.bfloat16).float()    # channels whose memories differ
        ids = tokens(60)
        want = O.forward(cfg, W, ids)[0]
        close(build(cfg, W, device, dtype)(torch.tensor([ids], device=device))[0], want, dtype, ALONE)
        for mistake in mistakes:
            assert float(position_errors(O.forward(cfg, W, ids, mistake=mistake)[0].float(), want).max()) > TOL[dtype], mistake


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("kw", [dict(), dict(width=65, vocab=101), dict(alpha=6.0, cap=2.0, eps=1e-2), dict(width=200, vocab=33)])
def test_whole_prompt_layer_by_layer(device, dtype, kw):
    cfg = mixed_config(**kw)
    W = O.random_weights(cfg, seed=2)
    ids = tokens(61, cfg["vocab"])
    want, streams = O.forward(cfg, W, ids)
    m, got = build(cfg, W, device, dtype), []
    close(m(torch.tensor([ids], device=device), collect=got)[0], want, dtype, WHOLE)
    assert len(got) == len(streams)
    for a, b in zip(got, streams):
        close(a[0], b, dtype, WHOLE)
    for mistake in ("no_gate", "no_decay"):
        assert float(position_errors(O.forward(cfg, W, ids, mistake=mistake)[0].float(), want).max()) > 1.5 * TOL[dtype], mistake


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("sizes", [[2] * 30 + [1], [61], [13, 8, 2, 21, 1, 1, 15], [1] * 61, [40] + [1] * 21, [3] * 20 + [1]])
def test_portions_and_token_by_token(device, dtype, sizes):
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    ids = tokens(61)
    close(run_portions(build(cfg, W, device, dtype), ids, sizes), O.forward(cfg, W, ids)[0], dtype, WHOLE)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_shared_keys_and_values(device, dtype):
    """A layer that shares another's cache holds nothing of its own, sees the keys as that cache holds them, and leaves them alone."""
    cfg = O.config([O.attention_spec(), O.lightning_spec(), O.attention_spec(heads=6, cap=2.0, scale=0.5, kv_from=0)], alpha=0.7)
    W = O.random_weights(cfg, seed=4)
    assert not any(n.startswith("l2.mix.k") or n.startswith("l2.mix.v") for n in W)
    m, ids = build(cfg, W, device, dtype), tokens(40)
    cache = m.make_cache(1, 40)
    assert cache.states[2]["k"].data_ptr() == cache.states[0]["k"].data_ptr() and cache.states[2]["v"].data_ptr() == cache.states[0]["v"].data_ptr()
    row = m.make_cache(3, 40).row(1)
    assert row.states[2]["k"].data_ptr() == row.states[0]["k"].data_ptr()
    want = O.forward(cfg, W, ids)[0]
    for sizes in ([40], [17, 1, 1, 21], [1] * 40):
        close(run_portions(m, ids, sizes), want, dtype, WHOLE)
    # the sharing layer's queries reach the first token: its own contribution disappears when layer 2 is cut off from it
    wrong = O.forward(cfg, W, ids, mistake="no_first")[0]
    assert float(position_errors(wrong.float(), want).max()) > 1.5 * TOL[dtype]


@pytest.mark.parametrize("device,dtype", EXACT)
def test_far_tokens_reach_through_every_mixer(device, dtype):
    """A change of the first token reaches the last position through the cache of the attention layers and through both kinds of state."""
    for layer in (O.attention_spec(), O.lightning_spec(decay=[0.999, 0.5, 1.0]), O.channel_delta_spec()):
        cfg = O.config([layer], alpha=0.5)
        W = O.random_weights(cfg, seed=4)
        for k in W:
            if k.endswith("A_log"):
                W[k] = torch.full_like(W[k], -6.0)   # slow decay: the state remembers
        m, ids = build(cfg, W, device, dtype), tokens(50)
        other = [(ids[0] + 1) % 104] + ids[1:]
        d = [float((run_portions(m, a, [20, 20, 10])[-1] - run_portions(m, b, [50])[-1]).abs().max()) for a, b in ((ids, ids), (ids, other))]
        assert d[0] < 1e-4 and d[1] > 1e-3, (layer["type"], d)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_batch_of_equal_prompts_against_each_alone(device, dtype):
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    m = build(cfg, W, device, dtype)
    rows = [tokens(53, seed=s) for s in range(3)]
    cache = m.make_cache(3, 60)
    ids = torch.tensor(rows, device=device)
    got = torch.cat([m(ids[:, :19], cache=cache), m(ids[:, 19:20], cache=cache), m(ids[:, 20:], cache=cache)], 1)
    for b, row in enumerate(rows):
        close(got[b], O.forward(cfg, W, row)[0], dtype, WHOLE)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_long_decoding(device, dtype):
    cfg = O.config([O.lightning_spec(decay=[0.9, 0.99, 0.999]), O.attention_spec(dim=64, vdim=64), O.channel_delta_spec(conv=4)], width=40)
    W = O.random_weights(cfg, seed=6)
    ids = tokens(300)
    want = O.forward(cfg, W, ids)[0]
    m = build(cfg, W, device, dtype)
    close(run_portions(m, ids, [3] + [1] * 297), want, dtype, WHOLE)
    close(run_portions(m, ids, [131, 2, 167]), want, dtype, WHOLE)


# ------------------------------------------------------------------------------------------------ pools, scheduler, entry points
@pytest.mark.parametrize("device,dtype", PLACES)
def test_pool_rows_are_reused_and_do_not_disturb_each_other(device, dtype):
    """Unequal requests interleaved on two rows: portions of one while the other decodes, rows closed and opened again."""
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    m = build(cfg, W, device, dtype)
    pool = SequencePool(m, 2, 64)
    reqs = {n: tokens(n, seed=n) for n in (30, 17, 2, 45, 64)}
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
    s64 = pool.open()
    extend(64, s64, 0, 64, False)                # a full row that sits out the other row's decode steps
    decode(45, s45, 20, 32)
    pool.close(s64)
    s2 = pool.open()
    extend(2, s2, 0, 2, False)
    decode(45, s45, 32, 45)
    for n in reqs:
        close(torch.cat(got[n]), want[n], dtype, WHOLE)


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
    want = [greedy_oracle(cfg, W, p, 8) for p in prompts]
    params = SamplingParams.from_mode("greedy", max_new_tokens=8)
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
    prompts = [tokens(n, seed=n) for n in (4, 39, 11)]
    outs = ContinuousBatcher(GenerationEngine(m), max_batch=2, max_len=64, prefill_chunk=17).run(prompts, 16)
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
            close(runner.step(rec), want[[at + k for k in keep]], dtype)   # (few positions: the mean is close to the worst)
            at += n
    assert runner.pool.available == 2


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program(tmp_path, dtype):
    cfg = mixed_config()
    W = O.random_weights(cfg, seed=2)
    O.save_model(str(tmp_path / "m"), cfg, W)
    ids = tokens(42)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:40], "want": [3, 9]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": ids[40:41], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": ids[41:], "want": [0]}], "end": ["x"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "48"],
                       input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = O.forward(cfg, W, ids)[0]
    for step, at in ((0, [3, 9]), (2, [41])):
        raw = torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32).view(len(at), -1)
        close(raw, want[at], getattr(torch, dtype))
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


# ------------------------------------------------------------------------------------------------ configuration, folders
def test_configuration_round_trip_and_errors(tmp_path):
    d = json.loads(json.dumps(mixed_config()))
    cfg = NemipelConfig.from_dict(d)
    assert NemipelConfig.from_dict(cfg.to_dict()) == cfg
    changes = [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][1]["mixer"].pop("heads"), lambda c: c["layers"][1]["mixer"].update(kv_heads=3),
               lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18),
               lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 1.5, 0.1]),
               lambda c: c["layers"][3]["mixer"].update(kv_from=0), lambda c: c["layers"][3]["mixer"].update(kv_from=6), lambda c: c["layers"][7]["mixer"].update(kv_from=3),
               lambda c: c["layers"][3]["mixer"].update(kv_heads=3), lambda c: c["layers"][2]["mlp"].update(kind="other"), lambda c: c["layers"][5]["mixer"].update(dim=300)]
    for change in changes:
        bad = json.loads(json.dumps(d))
        change(bad)
        with pytest.raises(ValueError):
            NemipelConfig.from_dict(bad)
    W = O.random_weights(mixed_config())
    for name, error in (("l0.norm1", "missing"), ("l2.mix.a1", "missing")):
        with pytest.raises(ValueError, match=error):
            build(d, {k: v for k, v in W.items() if k != name}, "cpu", torch.float32)
    with pytest.raises(ValueError, match="unexpected"):
        build(d, {**W, "l3.mix.k": W["l1.mix.k"]}, "cpu", torch.float32)
    model = build(d, W, "cpu", torch.float32)
    assert (model.mixers[2].s.decay_rank, model.mixers[2].s.gate_rank) == (10, 6)
    assert model.num_parameters() == sum(v.numel() for v in W.values())
    assert Nemipel.random(cfg, torch.float32, "cpu")(torch.tensor([[1, 2, 3]])).shape == (1, 3, 104)
