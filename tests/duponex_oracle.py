"""Plain restatement of the Duponex decoder for the tests: one function per mechanism, whole sequences, no cache, no
batching, nothing imported from the package. ``dt`` is the arithmetic type (float64 by default)."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def relu_squared(z):
    return torch.clamp(z, min=0) ** 2


def chunk_visible(n: int, size: int) -> torch.Tensor:
    """[n, n] bool: row i may look at column j (not after it, and in the same block of ``size`` positions)."""
    i = torch.arange(n)
    return (i[None, :] <= i[:, None]) & (torch.div(i, size, rounding_mode="floor")[None, :] == torch.div(i, size, rounding_mode="floor")[:, None])


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, t, p, cfg, eps, v_first):
    """One mixer on [n, width] rows. ``t``: tensor getter; returns (result, this layer's unmixed values)."""
    n = h.shape[0]
    H, G, dk, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = (h @ t(p + "q").T + t(p + "q.b")).view(n, H, dk)
    k = (h @ t(p + "k").T + t(p + "k.b")).view(n, G, dk)
    v = (h @ t(p + "v").T + t(p + "v.b")).view(n, G, dv)
    own = v
    q, k = rms(q, eps), rms(k, eps)
    if cfg.get("v_mix") and v_first is not None:
        v = mix_values(v, v_first, t(p + "vmix"))
    see = chunk_visible(n, cfg["mask"]["size"])
    out = torch.empty(n, H, dv, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * cfg["scale"]
        w = torch.softmax(s.masked_fill(~see, -math.inf), -1)
        out[:, a] = w @ v[:, g]
    gated = out.reshape(n, H * dv) * torch.sigmoid(h @ t(p + "g").T)
    return gated @ t(p + "o").T + t(p + "o.b"), own


def feed_forward(h, t, p):
    return relu_squared(h @ t(p + "up").T) @ t(p + "down").T


def stream_read(xs, w_in):
    return torch.einsum("snd,s->nd", xs, w_in)


def stream_write(xs, y, mix, w_out, m):
    """xs [streams, n, width]; ``mix[a, b]`` carries stream a into stream b."""
    return torch.einsum("ab,and->bnd", mix, xs) + m * w_out[:, None, None] * y[None]


def forward(config: dict, tensors: dict, tokens, dt=torch.float64):
    """Logits [n, vocab] of a whole sequence and the summed residual after every layer [layers, n, width]."""
    t = lambda name: tensors[name].to(dt)
    eps, m, streams = config["norm"]["eps"], config["residual_mult"], config["streams"]
    e = t("embed")[torch.as_tensor(tokens)] * config["embedding"]["scale"]
    xs = e[None].repeat(streams, 1, 1)
    v_first, after = None, []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        u = stream_read(xs, t(p + "hc1.in"))
        y, own = attention(rms(u, eps) * t(p + "norm1"), t, p + "mix.", layer["mixer"], eps, v_first)
        if layer["mixer"].get("v_mix") and v_first is None:
            v_first = own
        xs = stream_write(xs, y * t(p + "ls1"), t(p + "hc1.mix"), t(p + "hc1.out"), m)
        if layer.get("mlp") is not None:
            u = stream_read(xs, t(p + "hc2.in"))
            y = feed_forward(rms(u, eps) * t(p + "norm2"), t, p + "mlp.")
            xs = stream_write(xs, y * t(p + "ls2"), t(p + "hc2.mix"), t(p + "hc2.out"), m)
        after.append(xs.sum(0))
    x = rms(xs.sum(0), eps) * t("final.norm")
    return x @ t("head").T, torch.stack(after)


# ------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------
def mixer(heads=4, kv_heads=2, dim=32, vdim=24, size=50, scale=0.3, v_mix=True):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale, "v_mix": v_mix}


def layer(ff=72, **kw):
    return {"type": "attention", "mixer": mixer(**kw), "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=104, vocab=198, streams=2, residual_mult=0.6, scale=3.0, eps=1e-5):
    return {"architecture": "Duponex", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps},
            "residual_mult": residual_mult, "streams": streams, "vocab": vocab, "width": width}


def tensors(cfg, seed=0):
    """Random weights (BF16 values) in which no factor is one and no matrix symmetric."""
    g = torch.Generator().manual_seed(seed)
    w, s = cfg["width"], cfg["streams"]
    rn = lambda *shape: torch.randn(*shape, generator=g)
    out = {"embed": rn(cfg["vocab"], w), "head": rn(cfg["vocab"], w) / w ** 0.5, "final.norm": 1 + 0.2 * rn(w)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        q, k, v, o = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
        for name, n in (("q", q), ("k", k), ("v", v)):
            out[p + "mix." + name] = rn(n, w) / w ** 0.5
            out[p + f"mix.{name}.b"] = 0.4 * rn(n)
        out[p + "mix.g"] = rn(o, w) / w ** 0.5
        out[p + "mix.o"], out[p + "mix.o.b"] = rn(w, o) / o ** 0.5, 0.3 * rn(w)
        if m["v_mix"]:
            out[p + "mix.vmix"] = torch.sigmoid(rn(()))
        subs = [1]
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            out[p + "mlp.up"], out[p + "mlp.down"] = rn(ff, w) / w ** 0.5, rn(w, ff) / ff ** 0.5
            subs.append(2)
        for n in subs:
            out[p + f"norm{n}"], out[p + f"ls{n}"] = 1 + 0.2 * rn(w), 1 + 0.3 * rn(w)
            out[p + f"hc{n}.in"], out[p + f"hc{n}.out"] = (1 + 0.4 * rn(s)) / s, 1 + 0.4 * rn(s)
            out[p + f"hc{n}.mix"] = 0.8 * torch.eye(s) + 0.15 * rn(s, s)
    return {n: t.to(torch.bfloat16) for n, t in out.items()}
