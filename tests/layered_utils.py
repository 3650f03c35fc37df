"""Helpers shared by the tests of layer-listed decoders (``test_vimodra.py``, ``test_nemipel.py``)."""
import pytest
import torch

gpu = pytest.mark.gpu
PLACES = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="gpu-fp32", marks=gpu),
          pytest.param("cuda", torch.bfloat16, id="gpu-bf16", marks=gpu)]
EXACT = PLACES[:2]
# root-mean-square error of the logits of a position over the root mean square of all logits: the worst position may reach TOL, the
# mean over the positions 40 % of it (random bf16 models scatter: near ties of the scores and large gates amplify a rounding)
TOL = {torch.float32: 1e-4, torch.bfloat16: 0.12}


def position_errors(got, want):
    want = want.float()
    d = got.float().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


def close(got, want, dtype, factor=1.0):
    e = position_errors(got, want)
    assert float(e.max()) < factor * TOL[dtype], f"worst position {int(e.flatten().argmax())}: {float(e.max()):.3g}"
    assert float(e.mean()) < factor * TOL[dtype] * 0.4, f"mean {float(e.mean()):.3g}"


def tokens(n, vocab=104, seed=1):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_portions(model, ids, sizes):
    """Logits of every position when the tokens come in portions of these sizes."""
    dev = model.embed.device
    cache, out, at = model.make_cache(1, len(ids)), [], 0
    for n in sizes:
        part = torch.tensor([ids[at:at + n]], device=dev)
        out.append(model(part, cache=cache)[0].float().cpu())
        at += n
    assert at == len(ids)
    return torch.cat(out)
