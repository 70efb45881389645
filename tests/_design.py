"""What the tests of the layer-list designs share: forms to run in, tolerances, small checkpoints, feeding in portions."""
import json

import pytest
import torch

from flyingfish_b200.api import Model
from flyingfish_b200.config import Settings
from flyingfish_b200.engine.engine import Span
from flyingfish_b200.loaders.safetensors_io import save_safetensors

GPU = pytest.mark.gpu
FORMS = [("cpu", "fp32"), pytest.param("cuda", "fp32", marks=GPU), pytest.param("cuda", "bf16", marks=GPU)]
each_form = pytest.mark.parametrize("device,dtype", FORMS)
TORCH = {"fp32": torch.float32, "bf16": torch.bfloat16}
# root mean square of a row's logit error over the oracle's, per row; the worst row must stay below
LIMIT = {"fp32": 5e-5, "bf16": 6e-2}


def close(got, want, dtype, what="", limit=None):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    err = ((got - want) ** 2).mean(-1).sqrt() / (want ** 2).mean(-1).sqrt().clamp(min=1e-3)
    assert err.max() <= (limit or LIMIT[dtype]), f"{what}: error {err.max().item():.3g} at row {int(err.argmax())}"


def write(tmp_path, cfg, tensors, name="m"):
    d = tmp_path / name
    d.mkdir()
    (d / "config.json").write_text(json.dumps(cfg))
    save_safetensors(d / "model.safetensors", tensors)
    return str(d)


def load(path, device, dtype, capacity=320, max_batch=4, **kw):
    return Model.load(path, Settings(capacity=capacity, max_batch=max_batch, dtype=dtype, **kw), device=device)


def ids(n, vocab=198, seed=1):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def feed_in_cuts(engine, tokens, cuts, seq=None):
    """Logits of all tokens, fed in portions of the given sizes (the last size repeats)."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(cuts[min(i, len(cuts) - 1)], len(tokens) - at)
        part = tokens[at: at + n]
        if seq is None:
            seq = engine.add_sequence(part)
        out.append(engine.feed([Span(seq, part, list(range(n)))]).float().cpu())
        at, i = at + n, i + 1
    return torch.cat(out), seq


def paged(device, dt, hkv, dk, dv, ctx, seed):
    """Keys / values of sequences laid out over shuffled blocks, and the same rows as plain tensors."""
    g = torch.Generator().manual_seed(seed)
    need = [(c + 63) // 64 for c in ctx]
    nb = sum(need) + 3
    perm = torch.randperm(nb, generator=g).tolist()
    bt = torch.zeros(len(ctx), max(need), dtype=torch.int32)
    kc, vc = torch.randn(nb, hkv, 64, dk, generator=g).to(dt), torch.randn(nb, hkv, 64, dv, generator=g).to(dt)
    for b, n in enumerate(need):
        for j in range(n):
            bt[b, j] = perm.pop()
    rows = lambda cache, b, c: torch.cat([cache[int(bt[b, j])] for j in range((c + 63) // 64)], 1)[:, :c].double()
    return kc, vc, bt, [rows(kc, b, c) for b, c in enumerate(ctx)], [rows(vc, b, c) for b, c in enumerate(ctx)]
