"""Plain restatement of the Rudorax decoder for the tests: one function per mechanism, whole sequences, no cache, no batching,
nothing imported from the package. ``dt`` is the arithmetic type (float64 by default)."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_one(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def window_visible(n: int, size: int) -> torch.Tensor:
    """[n, n] bool: row i may look at itself and the ``size - 1`` columns before it."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < size)


def yarn_frequencies(rot):
    """(angle per position of every pair, factor of cos and sin), in double precision."""
    dims, base = rot["dims"], float(rot["base"])
    s = rot.get("scaling")
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if s is None:
        return torch.tensor(plain, dtype=torch.float64), 1.0

    def place(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(place(s["fast"])), 0), min(math.ceil(place(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1.0


def rotate_pairs(x, rot, first=0):
    """x [n, heads, dim] at positions first, first + 1, ...: neighbours (2i, 2i + 1) of the first ``dims`` elements turn."""
    freq, amp = yarn_frequencies(rot)
    a = torch.arange(first, first + x.shape[0], dtype=torch.float64)[:, None] * freq
    c, s = (torch.cos(a) * amp).to(x.dtype)[:, None], (torch.sin(a) * amp).to(x.dtype)[:, None]
    out = x.clone()
    u, v = x[..., 0: rot["dims"]: 2], x[..., 1: rot["dims"]: 2]
    out[..., 0: rot["dims"]: 2] = u * c - v * s
    out[..., 1: rot["dims"]: 2] = v * c + u * s
    return out


def softmax_with_sink(s, sink):
    """Rows of scores and one extra logit that takes weight and gives nothing."""
    full = torch.cat([s, sink.expand(s.shape[0], 1)], -1)
    return torch.softmax(full, -1)[:, :-1]


def attention(h, t, p, cfg, eps):
    n = h.shape[0]
    H, G, dk, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = rms((h @ t(p + "q").T).view(n, H, dk), eps) * t(p + "q.norm")
    k = rms((h @ t(p + "k").T).view(n, G, dk), eps) * t(p + "k.norm")
    v = (h @ t(p + "v").T).view(n, G, dv)
    q, k = rotate_pairs(q, cfg["rot"]), rotate_pairs(k, cfg["rot"])
    see = window_visible(n, cfg["mask"]["size"])
    sink = t(p + "sink")
    out = torch.empty(n, H, dv, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * cfg["scale"]
        out[:, a] = softmax_with_sink(s.masked_fill(~see, -math.inf), sink[a]) @ v[:, g]
    return out.reshape(n, H * dv) @ t(p + "o").T


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def matrix_memory(q, k, v, i, f):
    """The recurrence, token by token. q, k [n, H, dk] (q scaled), v [n, H, dv], i, f [n, H] logarithms -> [n, H, dv]."""
    n, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype)
    nrm = torch.zeros(H, dk, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = torch.empty_like(v)
    for t in range(n):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        nrm = keep[:, None] * nrm + add[:, None] * k[t]
        m = new
        den = torch.maximum((nrm * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hkv,hk->hv", S, q[t]) / den[:, None]
    return out


def mlstm(h, t, p, cfg, eps):
    n = h.shape[0]
    H, dk, dv, cap = cfg["heads"], cfg["dim"], cfg["vdim"], cfg["gate_cap"]
    q = (h @ t(p + "q").T).view(n, H, dk) * dk ** -0.5
    k = (h @ t(p + "k").T).view(n, H, dk)
    v = (h @ t(p + "v").T).view(n, H, dv)
    i = capped(h @ t(p + "i").T + t(p + "i.b"), cap)
    f = torch.nn.functional.logsigmoid(capped(h @ t(p + "f").T + t(p + "f.b"), cap))
    o = rms(matrix_memory(q, k, v, i, f), eps).reshape(n, H * dv)
    return (o * t(p + "norm") * torch.sigmoid(h @ t(p + "g").T)) @ t(p + "o").T


def gated_silu(h, t, p):
    g = h @ t(p + "gate").T
    return (g * torch.sigmoid(g) * (h @ t(p + "up").T)) @ t(p + "down").T


MARGINS: list[float] = []        # distance between the last choice and the first refused one, of every choice made


def choose_experts(h, t, p, top):
    """(ids [n, top], weights [n, top]): the bias moves the choice, not the weights."""
    s = torch.softmax(h @ t(p + "router").T, -1)
    ordered = torch.sort(s + t(p + "correction"), dim=-1, descending=True).values
    if top < ordered.shape[1]:
        MARGINS.append(float((ordered[:, top - 1] - ordered[:, top]).min()))
    ids = torch.sort(s + t(p + "correction"), dim=-1, descending=True, stable=True).indices[:, :top]
    w = s.gather(1, ids)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20)


def mixture(h, t, p, cfg):
    r = cfg["router"]
    ids, w = choose_experts(h, t, p, r["top"])
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r["identity"]):
        rows, at = torch.nonzero(ids == e, as_tuple=True)
        if len(rows):
            y = h[rows] if e >= r["experts"] else gated_silu(h[rows], t, p + f"e{e}.")
            out[rows] += w[rows, at][:, None] * y
    return out + gated_silu(h, t, p + "shared.") if cfg.get("shared") else out


def run_order(config):
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(config: dict, tensors: dict, tokens, dt=torch.float64):
    """Logits [n, vocab] of a whole sequence and the residual after every layer run [runs, n, width]."""
    t = lambda name: tensors[name].to(dt)
    eps = config["norm"]["eps"]
    x = t("embed")[torch.as_tensor(tokens)] * config["embedding"]["scale"]
    after = []
    for i in run_order(config):
        layer, p = config["layers"][i], f"l{i}."
        mix = {"attention": attention, "mlstm": mlstm}[layer["type"]]
        y = mix(norm_around_one(x, t(p + "norm1"), eps), t, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + mixture(norm_around_one(x, t(p + "norm2"), eps), t, p + "mlp.", layer["mlp"])
        x = x + y
        after.append(x)
    z = norm_around_one(x, t("final.norm"), eps) @ t("head").T
    cap = config.get("logit_softcap")
    return capped(z, cap) if cap else z, torch.stack(after)


# ------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------
def rot(dims=16, base=5000.0, factor=3.0, original=300, fast=20.0, slow=2.0):
    return {"base": base, "dims": dims, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}


def moe(ff=40, experts=6, identity=2, top=3, shared=56):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}, "shared": {"ff": shared}}


_MOE = object()


def attn_layer(heads=4, kv_heads=2, dim=32, vdim=24, size=50, scale=0.3, turn=None, mlp=_MOE):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
            "scale": scale, "rot": turn or rot(dims=min(16, dim))}, "mlp": moe() if mlp is _MOE else mlp}


def mlstm_layer(heads=3, dim=24, vdim=40, gate_cap=7.0, mlp=_MOE):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}, "mlp": moe() if mlp is _MOE else mlp}


def config(layers, width=104, vocab=198, scale=3.0, eps=1e-5, softcap=9.0, loop=None):
    return {"architecture": "Rudorax", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps},
            "loop": loop and {"start": loop[0], "stop": loop[1], "times": loop[2]}, "logit_softcap": softcap, "vocab": vocab, "width": width}


CLASSES = 5


def tensors(cfg, seed=0):
    """Random weights (BF16 values) in which every mechanism counts. The experts a token gets hang on its class alone (its number
    modulo ``CLASSES``): the last channels carry the class and no layer writes to them, so that no choice is a close call which
    16-bit rounding could turn."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]
    rn = lambda *shape: torch.randn(*shape, generator=g)
    lin = lambda o, i, gain=1.0: gain * rn(o, i) / i ** 0.5

    def writes(i):
        m = lin(w, i)
        m[-CLASSES:] = 0.0
        return m
    out = {"embed": rn(cfg["vocab"], w) / cfg["embedding"]["scale"], "head": lin(cfg["vocab"], w, 3.0), "final.norm": 0.2 * rn(w)}
    out["embed"][:, -CLASSES:] = 0.0
    out["embed"][torch.arange(cfg["vocab"]), w - CLASSES + torch.arange(cfg["vocab"]) % CLASSES] = 4.0 / cfg["embedding"]["scale"]
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", l["mixer"]
        out[f"l{i}.norm1"] = 0.2 * rn(w)
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        out.update({p + "q": lin(H * dk, w), p + "k": lin(G * dk, w), p + "v": lin(G * dv, w), p + "o": writes(H * dv)})
        if l["type"] == "attention":
            out.update({p + "q.norm": 1 + 0.3 * rn(dk), p + "k.norm": 1 + 0.3 * rn(dk), p + "sink": 1.0 + 0.7 * rn(H)})
        else:
            out.update({p + "g": lin(H * dv, w), p + "norm": 1 + 0.3 * rn(H * dv), p + "i": lin(H, w, 2.0), p + "i.b": 0.5 * rn(H) - 1.0,
                        p + "f": lin(H, w, 2.0), p + "f.b": 0.5 * rn(H) + 3.0})
        if l.get("mlp") is not None:
            f = l["mlp"]
            p, r = f"l{i}.mlp.", f["router"]
            out[f"l{i}.norm2"] = 0.2 * rn(w)
            n = r["experts"] + r["identity"]
            out[p + "router"] = torch.zeros(n, w)
            always = int(torch.randint(0, n, (1,), generator=g))                # the output that the bias puts into every choice
            others = torch.tensor([j for j in range(n) if j != always], dtype=torch.long)
            for c in range(CLASSES):                      # a class's own outputs, the rest well below, the biased one anywhere
                level = torch.where(torch.arange(n - 1) < r["top"] - 1, 1.6 + 0.1 * rn(n - 1), -0.4 + 0.1 * rn(n - 1))
                out[p + "router"][others[torch.randperm(n - 1, generator=g)], w - CLASSES + c] = level
                out[p + "router"][always, w - CLASSES + c] = 2.0 * torch.rand((), generator=g) - 0.4
            out[p + "correction"] = 0.004 * rn(n)
            out[p + "correction"][always] = 2.0
            names = [(f"e{e}.", f["expert"]["ff"]) for e in range(r["experts"])] + ([("shared.", f["shared"]["ff"])] if f.get("shared") else [])
            for name, ff in names:
                out.update({p + name + "gate": lin(ff, w), p + name + "up": lin(ff, w), p + name + "down": writes(ff)})
    return {n: t.to(torch.bfloat16) for n, t in out.items()}
