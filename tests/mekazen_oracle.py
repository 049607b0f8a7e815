"""Plain, slow statement of the Mekazen decoder's equations in float64 / float32 tensors, one function per mechanism.

Nothing here is shared with the product code: sequences are processed whole (no cache), one at a time, and attention is a full
masked score matrix per head. ``forward`` returns the logits of every position and, when asked, the residual after every layer."""
import math

import torch


def rms_normalise(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms_normalise(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def frequencies(rot, dtype=torch.float64):
    """One angular frequency per rotated pair; long wavelengths are slowed down by the scaling, if there is one."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            turns = s["original"] / (2 * math.pi / f)              # how often the pair turns within the original length
            if turns < s["low"]:
                f = f / s["factor"]
            elif turns <= s["high"]:
                mix = (turns - s["low"]) / (s["high"] - s["low"])
                f = (1 - mix) * f / s["factor"] + mix * f
        out.append(f)
    return torch.tensor(out, dtype=dtype)


def rotate(x, positions, freq):
    """x [n, heads, D]: neighbouring dimensions (0, 1), (2, 3), ... turn by position times frequency; the rest stays."""
    r = 2 * len(freq)
    a = (positions.to(x.dtype).view(-1, 1) * freq.to(x.dtype)).unsqueeze(1)
    u, v = x[..., 0:r:2], x[..., 1:r:2]
    y = x.clone()
    y[..., 0:r:2] = u * torch.cos(a) - v * torch.sin(a)
    y[..., 1:r:2] = v * torch.cos(a) + u * torch.sin(a)
    return y


def chunk_visible(n, size):
    """[n, n] bool: query row i, key column j; both in the same chunk of ``size`` positions (None: one endless chunk)."""
    i, j = torch.arange(n).view(n, 1), torch.arange(n).view(1, n)
    ok = j <= i
    return ok if size is None else ok & (i // size == j // size)


def softmax_attention(q, k, v, scale, see):
    """q [n, H, D], k and v [n, G, D]; query head h reads key head h // (H // G)."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    heads = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~see, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        heads.append(e @ v[:, g] / e.sum(-1, keepdim=True))
    return torch.cat(heads, -1)


def attention(w, p, m, h, eps):
    n, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
    v = k.view(n, G, D)
    q = (rms_normalise(q, eps) * w[p + "q.norm"]).view(n, H, D)
    k = (rms_normalise(k, eps) * w[p + "k.norm"]).view(n, G, D)
    if m.get("rot"):
        f, pos = frequencies(m["rot"]), torch.arange(n)
        q, k = rotate(q, pos, f), rotate(k, pos, f)
    o = softmax_attention(q, k, v, m["scale"], chunk_visible(n, (m.get("mask") or {}).get("size")))
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated_mlp(w, p, h):
    z = h @ w[p + "gate"].T
    return (z * sigmoid(z) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def softcap(z, cap):
    return z if not cap else cap * torch.tanh(z / cap)


def forward(cfg, weights, tokens, dtype=torch.float64, residuals=None):
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    for i, L in enumerate(cfg["layers"]):
        l = f"l{i}."
        x = x + centred_norm(attention(w, l + "mix.", L["mixer"], centred_norm(x, w[l + "norm1"], eps), eps), w[l + "norm1b"], eps)
        if L["mlp"] is not None:
            x = x + centred_norm(gated_mlp(w, l + "mlp.", centred_norm(x, w[l + "norm2"], eps)), w[l + "norm2b"], eps)
        if residuals is not None:
            residuals.append(x)
    return softcap(centred_norm(x, w["final.norm"], eps) @ w["head"].T, cfg.get("logit_softcap"))


def random_weights(cfg, seed=0, dtype=torch.float32):
    """Seeded weights with every tensor of ``cfg``, scaled so that each mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)

    def lin(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * s * i ** -0.5

    def near(n, c, s):
        return c + s * torch.randn(n, generator=g)
    E = cfg["width"]
    w = {"embed": torch.randn(cfg["vocab"], E, generator=g), "final.norm": near(E, 0, 0.2), "head": lin(cfg["vocab"], E, 6.0)}
    for i, L in enumerate(cfg["layers"]):
        l, m = f"l{i}.", L["mixer"]
        H, G, D, p = m["heads"], m["kv_heads"], m["dim"], l + "mix."
        for q in ((1, 2) if L["mlp"] is not None else (1,)):
            w[f"{l}norm{q}"], w[f"{l}norm{q}b"] = near(E, 0, 0.2), near(E, 0, 0.2)
        w[p + "q"], w[p + "k"], w[p + "g"], w[p + "o"] = lin(H * D, E), lin(G * D, E), lin(H * D, E), lin(E, H * D)
        w[p + "q.norm"], w[p + "k.norm"] = near(H * D, 1.3, 0.2), near(G * D, 1.3, 0.2)
        if L["mlp"] is not None:
            F = L["mlp"]["ff"]
            w[l + "mlp.gate"], w[l + "mlp.up"], w[l + "mlp.down"] = lin(F, E), lin(F, E), lin(E, F)
    return {n: t.to(torch.bfloat16).to(dtype) for n, t in w.items()}
