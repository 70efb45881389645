"""Plain restatement of the Kabavik decoder for the tests: one function per mechanism, whole sequences, no cache, no batching,
nothing imported from the package. ``dt`` is the arithmetic type (float64 by default)."""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------------------
# mechanisms
# ------------------------------------------------------------------------------------------
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def tanh_norm(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def visible(n: int, mask, first: int = 0) -> torch.Tensor:
    """[n, first + n] bool: what the row at position first + i may look at."""
    i, j = torch.arange(first, first + n)[:, None], torch.arange(first + n)[None, :]
    see = j <= i
    if mask:
        see = see & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return see


def linear_frequencies(rot):
    f = [float(rot["base"]) ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    s = rot.get("scaling")
    return torch.tensor(f, dtype=torch.float64) / (s["factor"] if s else 1.0), 1.0


def yarn_frequencies(rot):
    dims, base = rot["dims"], float(rot["base"])
    s = rot.get("scaling")
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return torch.tensor(plain, dtype=torch.float64), 1.0

    def place(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(place(s["fast"])), 0), min(math.ceil(place(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1.0


def _turned(x, freq, amp, first, pick_u, pick_v):
    a = torch.arange(first, first + x.shape[0], dtype=torch.float64)[:, None] * freq
    c, s = (torch.cos(a) * amp).to(x.dtype)[:, None], (torch.sin(a) * amp).to(x.dtype)[:, None]
    out = x.clone()
    u, v = x[..., pick_u], x[..., pick_v]
    out[..., pick_u] = u * c - v * s
    out[..., pick_v] = v * c + u * s
    return out


def rotate_halves(x, rot, first=0):
    """x [n, heads, dim] at positions first, first + 1, ...: element i of the first ``dims`` turns with element i + dims / 2."""
    freq, amp = linear_frequencies(rot)
    h = rot["dims"] // 2
    return _turned(x, freq, amp, first, slice(0, h), slice(h, 2 * h))


def rotate_pairs(x, rot, first=0):
    """Neighbours (2i, 2i + 1) turn."""
    freq, amp = yarn_frequencies(rot)
    return _turned(x, freq, amp, first, slice(0, rot["dims"], 2), slice(1, rot["dims"], 2))


def query_temperature(n, cfg, first=0):
    p = torch.arange(first, first + n, dtype=torch.float64)
    return 1.0 + cfg["coef"] * torch.log(torch.floor((p + 1.0) / cfg["every"]) + 1.0)


def attend(q, k, v, scale, see, cap=None):
    """q [n, H, dk], k [m, G, dk], v [m, G, dv] -> [n, H, dv]; query head h reads key head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    out = torch.empty(q.shape[0], H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        out[:, h] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g]
    return out


def biased(h, t, name):
    return h @ t(name).T + t(name + ".b")


# ------------------------------------------------------------------------------------------
# mixers
# ------------------------------------------------------------------------------------------
def windowed(h, t, p, cfg, eps, shared):
    """``shared``: (keys, values) of the layer this one borrows them from, or None. Returns the result and the layer's own pair."""
    n, H, G, dk, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = rms(biased(h, t, p + "q"), eps) * t(p + "q.norm")
    q = rotate_halves(q.view(n, H, dk), cfg["rot"])
    if shared is None:
        k = rms(biased(h, t, p + "k"), eps) * t(p + "k.norm")
        shared = rotate_halves(k.view(n, G, dk), cfg["rot"]), biased(h, t, p + "v").view(n, G, dv)
    o = attend(q, *shared, cfg["scale"], visible(n, cfg.get("mask")))
    return biased(o.reshape(n, H * dv), t, p + "o"), shared


def capped(h, t, p, cfg, eps, shared):
    n, H, G, dk, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = rms(biased(h, t, p + "q").view(n, H, dk), eps) * t(p + "q.norm")
    if shared is None:
        shared = rms(biased(h, t, p + "k").view(n, G, dk), eps) * t(p + "k.norm"), biased(h, t, p + "v").view(n, G, dv)
    if cfg.get("q_temp"):
        q = q * query_temperature(n, cfg["q_temp"]).to(q.dtype)[:, None, None]
    o = attend(q, *shared, cfg["scale"], visible(n, cfg.get("mask")), cfg.get("softcap"))
    return biased(o.reshape(n, H * dv), t, p + "o"), shared


def latent(h, t, p, cfg, eps, shared):
    n, H, dk, rd, dv, r = h.shape[0], cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    q = (h @ t(p + "q").T).view(n, H, dk + rd)
    down = h @ t(p + "dkv").T
    c = rms(down[:, :r], eps) * t(p + "dkv.norm")
    kr = rotate_pairs(down[:, None, r:], cfg["rot"]).expand(n, H, rd)
    k = torch.cat([(c @ t(p + "uk").T).view(n, H, dk), kr], -1)
    q = torch.cat([q[..., :dk], rotate_pairs(q[..., dk:], cfg["rot"])], -1)
    v = (c @ t(p + "uv").T).view(n, H, dv)
    o = attend(q, k, v, cfg["scale"], visible(n, cfg.get("mask")))
    o = o * torch.sigmoid(h @ t(p + "g").T)[..., None]
    return o.reshape(n, H * dv) @ t(p + "o").T, None


MIXERS = {"attention": windowed, "attention_2": capped, "latent_attention": latent}


def feed_forward(h, t, p):
    return (gelu_tanh(h @ t(p + "gate").T) * (h @ t(p + "up").T)) @ t(p + "down").T


def token_side(x, e, t, p, eps):
    y = (gelu_tanh(x @ t(p + "gate").T) * e) @ t(p + "proj").T
    return rms(y, eps) * t(p + "norm")


def forward(config: dict, tensors: dict, tokens, dt=torch.float64):
    """Logits [n, vocab] of a whole sequence and the residual after every layer [layers, n, width]."""
    t = lambda name: tensors[name].to(dt)
    norm = lambda x, name: tanh_norm(x, t(name + ".alpha"), t(name), t(name + ".b"))
    eps, m = config["norm"]["eps"], config["residual_mult"]
    ids = torch.as_tensor(tokens)
    x = t("embed")[ids] * config["embedding"]["scale"]
    side = config.get("token_side")
    after, kept = [], {}
    for i, layer in enumerate(config["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        src = mix.get("kv_from")
        y, kept[i] = MIXERS[layer["type"]](norm(x, p + "norm1"), t, p + "mix.", mix, eps, None if src is None else kept[src])
        x = x + m * norm(y, p + "norm1b")
        if layer.get("mlp") is not None:
            x = x + m * norm(feed_forward(norm(x, p + "norm2"), t, p + "mlp."), p + "norm2b")
        if side:
            d = side["dim"]
            x = x + m * token_side(x, t("side.embed")[ids][:, i * d: (i + 1) * d], t, p + "side.", eps)
        after.append(x)
    return norm(x, "final.norm") @ t("head").T * config["logit_scale"], torch.stack(after)


# ------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------
_FF = object()


def linear_rot(dims=12, base=4000.0, factor=3.0):
    return {"base": base, "dims": dims, "scaling": {"factor": factor}}


def yarn_rot(dims=8, base=700.0, factor=6.0, original=200, fast=24.0, slow=1.5):
    return {"base": base, "dims": dims, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}


def _ff(mlp, ff=88):
    return {"kind": "dense", "ff": ff} if mlp is _FF else mlp


def window_layer(heads=6, kv_heads=2, dim=40, vdim=24, size=50, keep=3, scale=0.21, turn=None, kv_from=None, mlp=_FF):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": turn or linear_rot(),
         "mask": {"size": size, "keep_first": keep}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": _ff(mlp)}


def capped_layer(heads=4, kv_heads=2, dim=48, vdim=32, scale=0.4, softcap=5.0, coef=0.4, every=37, mlp=_FF):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                             "softcap": softcap, "q_temp": {"coef": coef, "every": every}}, "mlp": _ff(mlp)}


def latent_layer(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=56, size=45, scale=0.3, turn=None, mlp=_FF):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                                  "rot": turn or yarn_rot(dims=rot_dim), "mask": {"size": size}}, "mlp": _ff(mlp)}


def config(layers, width=104, vocab=198, scale=1.7, eps=2e-5, mult=0.6, side=20, logit_scale=0.8):
    return {"architecture": "Kabavik", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult,
            "token_side": {"dim": side} if side else None, "logit_scale": logit_scale, "vocab": vocab, "width": width}


def tensors(cfg, seed=0):
    """Random weights (BF16 values) in which every mechanism counts."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]
    rn = lambda *shape: torch.randn(*shape, generator=g)
    lin = lambda o, i, gain=1.0: gain * rn(o, i) / i ** 0.5
    out = {"embed": rn(cfg["vocab"], w) / cfg["embedding"]["scale"], "head": lin(cfg["vocab"], w, 3.0)}

    def norm(name, alpha=0.7):
        out.update({name: 1.0 + 0.2 * rn(w), name + ".b": 0.1 * rn(w), name + ".alpha": alpha + 0.1 * rn(1)[0]})

    def proj(name, o, i):
        out.update({name: lin(o, i), name + ".b": 0.3 * rn(o)})
    norm("final.norm")
    side = cfg.get("token_side")
    if side:
        out["side.embed"] = rn(cfg["vocab"], len(cfg["layers"]) * side["dim"])
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", l["mixer"]
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l.get("mlp") is not None else ()):
            norm(f"l{i}.{n}")
        if l["type"] == "latent_attention":
            r, rd = m["kv_rank"], m["rot_dim"]
            out.update({p + "q": lin(H * (dk + rd), w), p + "dkv": lin(r + rd, w), p + "dkv.norm": 1.0 + 0.3 * rn(r), p + "uk": lin(H * dk, r),
                        p + "uv": lin(H * dv, r), p + "g": lin(H, w, 2.0), p + "o": lin(w, H * dv)})
        else:
            G, whole = m["kv_heads"], l["type"] == "attention"
            proj(p + "q", H * dk, w)
            out[p + "q.norm"] = 1.0 + 0.3 * rn(H * dk if whole else dk)
            if m.get("kv_from") is None:
                proj(p + "k", G * dk, w)
                proj(p + "v", G * dv, w)
                out[p + "k.norm"] = 1.0 + 0.3 * rn(G * dk if whole else dk)
            proj(p + "o", w, H * dv)
        if l.get("mlp") is not None:
            f, p = l["mlp"]["ff"], f"l{i}.mlp."
            out.update({p + "gate": lin(f, w), p + "up": lin(f, w), p + "down": lin(w, f)})
        if side:
            p = f"l{i}.side."
            out.update({p + "gate": lin(side["dim"], w), p + "proj": lin(w, side["dim"]), p + "norm": 0.5 + 0.2 * rn(w)})
    return {n: t.to(torch.bfloat16) for n, t in out.items()}
