"""Plain restatement of the Bazulorn decoder for the tests: one function per mechanism, whole sequences, no cache, no batching,
nothing imported from the package. ``dt`` is the arithmetic type (float64 by default)."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_rows(ids, cfg):
    """Row of the second table for every token: a mix of the token before and the token itself; the first token has a row of its own."""
    out = []
    for i, t in enumerate(ids):
        out.append(cfg["buckets"] if i == 0 else (ids[i - 1] * cfg["mul_prev"] + t * cfg["mul_cur"]) % cfg["buckets"])
    return out


def embedding(ids, t, cfg, eps):
    x = t("embed")[ids] + t("bigram")[bigram_rows(ids, cfg["embedding"]["bigram"])]
    return rms(x, eps) * t("embed.norm")


def causal_conv(x, w, bias=None):
    """x [n, channels], w [channels, taps], the last column weighs the current row; zeros before the first row."""
    n, taps = x.shape[0], w.shape[1]
    full = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    y = sum(full[j: j + n] * w[:, j] for j in range(taps))
    return y if bias is None else y + bias


def window_visible(n, size):
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < size)


def softmax_with_one(s):
    """exp(s) / (1 + sum exp(s)) over the last dimension."""
    m = s.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def talking_attention(q, k, v, scale, size, talk):
    """q [n, H, dk], k, v [n, G, ..] (values already normed) -> [n, H, dv]: every head's weights, mixed over the heads, on its own values."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    see = window_visible(n, size)
    w = torch.stack([softmax_with_one(((q[:, h] @ k[:, h // (H // G)].T) * scale).masked_fill(~see, -math.inf)) for h in range(H)])
    mixed = torch.einsum("hg,gij->hij", talk, w)
    return torch.stack([mixed[h] @ v[:, h // (H // G)] for h in range(H)], 1)


def left(h, t, p, cfg, eps):
    n, H, G, dk, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    proj = lambda name: h @ t(p + name).T + t(p + name + ".b")
    v = rms(proj("v").view(n, G, dv), eps)
    o = talking_attention(proj("q").view(n, H, dk), proj("k").view(n, G, dk), v, cfg["scale"], cfg["mask"]["size"], t(p + "talk"))
    return o.reshape(n, H * dv) @ t(p + "o").T


def state_space(x, B, C, dt, a, D):
    """x [n, H, dv], B, C [n, H, N], dt [n, H], a [H] (negative), D [H] -> [n, H, dv], token by token."""
    n, H, dv = x.shape
    S = torch.zeros(H, B.shape[2], dv, dtype=x.dtype)
    out = torch.empty_like(x)
    for i in range(n):
        S = torch.exp(a * dt[i])[:, None, None] * S + (dt[i][:, None] * B[i])[:, :, None] * x[i][:, None, :]
        out[i] = torch.einsum("hnv,hn->hv", S, C[i]) + D[:, None] * x[i]
    return out


def gated_group_norm(y, z, groups, w, eps):
    g = (y * silu(z)).view(y.shape[0], groups, -1)
    return rms(g, eps).reshape(y.shape) * w


def right(h, t, p, cfg, eps):
    n, H, dv, N, G = h.shape[0], cfg["heads"], cfg["vdim"], cfg["state"], cfg["groups"]
    inner = H * dv
    z, x, B, C, dt = torch.split(h @ t(p + "in").T, [inner, inner, G * N, G * N, H], -1)
    xbc = silu(causal_conv(torch.cat([x, B, C], -1), t(p + "conv"), t(p + "conv.b")))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    spread = lambda m: m.view(n, G, N).repeat_interleave(H // G, 1)
    y = state_space(x.view(n, H, dv), spread(B), spread(C), softplus(dt + t(p + "dt_bias")), -torch.exp(t(p + "A_log")), t(p + "D"))
    return gated_group_norm(y.reshape(n, inner), z, cfg["norm_groups"], t(p + "norm"), eps) @ t(p + "o").T


def side_by_side(h, t, p, cfg, eps):
    l = rms(left(h, t, p + "left.", cfg["left"], eps), eps) * t(p + "left.out")
    r = rms(right(h, t, p + "right.", cfg["right"], eps), eps) * t(p + "right.out")
    return 0.5 * (l + r)


def delta_rule(q, k, v, beta, g):
    """q, k [n, H, dk], v [n, H, dv], beta [n, H], g [n, H, dk] decays -> [n, H, dv], token by token."""
    n, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype)
    out = torch.empty_like(v)
    for i in range(n):
        S = g[i][:, :, None] * S
        u = beta[i][:, None] * (v[i] - torch.einsum("hkv,hk->hv", S, k[i]))
        S = S + k[i][:, :, None] * u[:, None, :]
        out[i] = torch.einsum("hkv,hk->hv", S, q[i])
    return out


def channel_delta(h, t, p, cfg, eps):
    n, H, G, dk, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    conv = lambda name: silu(causal_conv(h @ t(p + name).T, t(p + name + ".conv")))
    spread = lambda m: m.repeat_interleave(H // G, 1)
    q = spread(unit(conv("q").view(n, G, dk)) * dk ** -0.5)
    k = spread(unit(conv("k").view(n, G, dk)))
    beta = torch.sigmoid(h @ t(p + "b").T)
    raw = (h @ t(p + "a1").T) @ t(p + "a2").T + t(p + "dt_bias")
    g = torch.exp(-torch.exp(t(p + "A_log"))[None, :, None] * softplus(raw).view(n, H, dk))
    o = rms(delta_rule(q, k, conv("v").view(n, H, dv), beta, g), eps) * t(p + "norm")
    gate = torch.sigmoid((h @ t(p + "g1").T) @ t(p + "g2").T)
    return (o.reshape(n, H * dv) * gate) @ t(p + "o").T


def dense_ff(h, t, p):
    return (gelu_tanh(h @ t(p + "gate").T) * (h @ t(p + "up").T)) @ t(p + "down").T


def expert_ff(h, t, p, limit):
    g, u = (h @ t(p + "gate").T).clamp(max=limit), (h @ t(p + "up").T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ t(p + "down").T


MARGINS: list[float] = []        # distance between the last choice and the first refused one, of every choice made


def choose_experts(h, t, p, top):
    z = h @ t(p + "router").T + t(p + "router.b")
    best = torch.topk(z, min(top + 1, z.shape[1]), -1)
    if z.shape[1] > top:
        MARGINS.extend((best.values[:, top - 1] - best.values[:, top]).tolist())
    return best.indices[:, :top], torch.softmax(best.values[:, :top], -1)


def experts(h, t, p, cfg):
    ids, w = choose_experts(h, t, p, cfg["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(cfg["router"]["experts"]):
        row, col = torch.nonzero(ids == e, as_tuple=True)
        if row.numel():
            out[row] += w[row, col, None] * expert_ff(h[row], t, p + f"e{e}.", cfg["expert"]["limit"])
    if cfg.get("shared"):
        out = out + expert_ff(h, t, p + "shared.", cfg["shared"]["limit"])
    return out


MIXERS = {"channel_delta": channel_delta, "parallel": side_by_side}


def forward(cfg, tensors, ids, dt=torch.float64):
    """(logits [n, vocab], residual after every layer [layers, n, width])."""
    t = lambda name: tensors[name].to(dt)
    eps = cfg["norm"]["eps"]
    x = embedding(list(ids), t, cfg, eps)
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms(x, eps) * t(p + "norm1")
        y = MIXERS[layer["type"]](h, t, p + "mix.", layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            y = y + (dense_ff(h, t, p + "mlp.") if mlp["kind"] == "dense" else experts(h, t, p + "mlp.", mlp))
        x = x + y
        after.append(x)
    return (rms(x, eps) * t("final.norm")) @ t("embed").T, torch.stack(after)


# ------------------------------------------------------------------------------------------
# configurations and weights for the tests
# ------------------------------------------------------------------------------------------
def moe(experts=6, top=3, ff=40, limit=1.5, shared=56, shared_limit=0.8):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit},
            "shared": {"ff": shared, "limit": shared_limit} if shared else None}


def dense(ff=88):
    return {"kind": "dense", "ff": ff}


def delta_layer(heads=4, kv_heads=2, dim=24, vdim=40, conv=4, mlp="moe", ranks=(20, 12)):
    """``ranks``: widths inside the matrix pairs of the decays and of the gate; a checkpoint's tensors have them, its configuration not."""
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": moe() if mlp == "moe" else mlp, "_ranks": ranks}


def pair_layer(heads=4, kv_heads=2, dim=32, vdim=24, size=50, scale=0.2, ssd=None, mlp="moe"):
    right = dict(heads=6, groups=3, state=20, vdim=28, conv=3, norm_groups=4)
    right.update(ssd or {})
    return {"type": "parallel", "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}},
                                          "right": right}, "mlp": moe() if mlp == "moe" else mlp}


def config(layers, width=104, vocab=198, eps=1e-5, buckets=61, mul_prev=13, mul_cur=5):
    return {"architecture": "Bazulorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}


def public(cfg):
    """The configuration as a checkpoint holds it."""
    return dict(cfg, layers=[{k: v for k, v in l.items() if k != "_ranks"} for l in cfg["layers"]])


def tensors(cfg, seed=0):
    """Seeded BF16 weights in which every mechanism counts. The first four channels hold the token's number modulo four, and nothing
    else writes there: the router reads mostly these, so that no choice of experts is close enough for rounding to turn it."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    t = {}
    rn = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i, f=1.0: f * rn(o, i) / i ** 0.5
    vec = lambda n, c=1.0, s=0.3: c + s * rn(n)

    def ff(p, f):
        t.update({p + "gate": lin(f, W, 1.5), p + "up": lin(f, W), p + "down": lin(W, f)})
    t.update({"embed": rn(cfg["vocab"], W), "bigram": rn(cfg["embedding"]["bigram"]["buckets"] + 1, W), "embed.norm": vec(W), "final.norm": vec(W)})
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        t[f"l{i}.norm1"] = vec(W)
        if layer["type"] == "channel_delta":
            ra, rg = layer["_ranks"]
            qk, v, k = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"] * m["dim"]
            for n, rows in (("q", qk), ("k", qk), ("v", v)):
                t.update({p + n: lin(rows, W), p + n + ".conv": 0.5 * rn(rows, m["conv"])})
            t.update({p + "b": lin(m["heads"], W), p + "A_log": vec(m["heads"], -1.5, 1.5), p + "norm": vec(m["vdim"]), p + "a1": lin(ra, W),
                      p + "a2": lin(k, ra), p + "dt_bias": vec(k, -2.0, 1.0), p + "g1": lin(rg, W), p + "g2": lin(v, rg), p + "o": lin(W, v)})
        else:
            a, r = m["left"], m["right"]
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                t.update({p + f"left.{n}": lin(rows, W), p + f"left.{n}.b": 0.3 * rn(rows)})
            o, inner, maps = a["heads"] * a["vdim"], r["heads"] * r["vdim"], r["groups"] * r["state"]
            t.update({p + "left.talk": torch.eye(a["heads"]) + 0.4 * rn(a["heads"], a["heads"]), p + "left.o": lin(W, o), p + "left.out": vec(W)})
            t.update({p + "right.in": lin(2 * inner + 2 * maps + r["heads"], W), p + "right.conv": 0.5 * rn(inner + 2 * maps, r["conv"]),
                      p + "right.conv.b": 0.3 * rn(inner + 2 * maps), p + "right.dt_bias": vec(r["heads"], -2.0, 1.0),
                      p + "right.A_log": vec(r["heads"], -1.5, 1.5), p + "right.D": vec(r["heads"]), p + "right.norm": vec(inner),
                      p + "right.o": lin(W, inner), p + "right.out": vec(W)})
        mlp, p = layer.get("mlp"), f"l{i}.mlp."
        if mlp is not None and mlp["kind"] == "dense":
            ff(p, mlp["ff"])
        elif mlp is not None:
            e = mlp["router"]["experts"]
            t.update({p + "router": lin(e, W, 0.05), p + "router.b": 0.1 * torch.rand(e, generator=g)})
            for c in range(4):
                t[p + "router"][:, c] = 0.4 * torch.randperm(e, generator=g)
            for j in range(e):
                ff(p + f"e{j}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                ff(p + "shared.", mlp["shared"]["ff"])
    t["embed"][:, :4] = 4.0 * torch.eye(4)[torch.arange(cfg["vocab"]) % 4]
    t["bigram"][:, :4] = 0.0
    for n, x in t.items():
        if n == "embed.norm" or n.endswith("norm1"):
            x[:4] = 1.0
        elif n.endswith((".o", ".down")):
            x[:4] = 0.0
    return {n: x.to(torch.bfloat16) for n, x in t.items()}
