"""Plain, slow statement of the Vebesun decoder's equations in float64 / float32 tensors, one function per mechanism.

Nothing here is shared with the product code: sequences are processed whole (no cache), one at a time, attention is a full
masked score matrix and the delta rule is a Python loop over tokens. ``forward`` returns the logits of every position and,
when asked, the sum of the residual streams after every layer run."""
import math

import torch


def rms_normalise(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    mu = x.mean(-1, keepdim=True)
    d = x - mu
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def silu(z):
    return z / (1 + torch.exp(-z))


def window_visible(n, size):
    """[n, n] bool: query row i, key column j; ``size`` None means every earlier token."""
    gap = torch.arange(n).view(n, 1) - torch.arange(n).view(1, n)
    ok = gap >= 0
    return ok if size is None else ok & (gap < size)


def latent_of(w, p, h, eps):
    return rms_normalise(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]


def latent_attention(w, p, cfg, h, eps):
    n, H, D, Dv = h.shape[0], cfg["heads"], cfg["dim"], cfg["vdim"]
    q = (h @ w[p + "q"].T).view(n, H, D)
    c = latent_of(w, p, h, eps)
    k = (c @ w[p + "uk"].T).view(n, H, D)
    v = (c @ w[p + "uv"].T).view(n, H, Dv)
    see = window_visible(n, (cfg.get("mask") or {}).get("size"))
    heads = []
    for a in range(H):
        s = (q[:, a] @ k[:, a].T) * cfg["scale"]
        s = s.masked_fill(~see, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        heads.append(e @ v[:, a] / e.sum(-1, keepdim=True))
    return torch.cat(heads, -1) @ w[p + "o"].T


def short_conv(x, taps):
    """x [n, channels], taps [channels, K]; the last tap multiplies the current token."""
    n, K = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for i in range(n):
        for t in range(K):
            j = i - (K - 1 - t)
            if j >= 0:
                out[i] += x[j] * taps[:, t]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_decay(w, p, heads, dim, h):
    """[n, heads, dim] factors in (0, 1)."""
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    sp = torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)
    return torch.exp(-torch.exp(w[p + "A_log"]).view(1, heads, 1) * sp.view(-1, heads, dim))


def delta_rule(q, k, v, beta, g, S=None):
    """q, k, g [n, H, D]; v [n, H, Dv]; beta [n, H] -> outputs [n, H, Dv] and the final state [H, D, Dv]."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if S is None else S.clone()
    out = []
    for i in range(n):
        S = S * g[i].unsqueeze(-1)
        u = beta[i].unsqueeze(-1) * (v[i] - torch.einsum("hdv,hd->hv", S, k[i]))
        S = S + k[i].unsqueeze(-1) * u.unsqueeze(1)
        out.append(torch.einsum("hdv,hd->hv", S, q[i]))
    return torch.stack(out), S


def channel_delta(w, p, cfg, h, eps):
    n, H, Hk, D, Dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    proj = {}
    for name in "qkv":
        proj[name] = silu(short_conv(h @ w[p + name].T, w[p + name + ".conv"]))
    head = torch.arange(H) // (H // Hk)
    q = (unit(proj["q"].view(n, Hk, D)) * D ** -0.5)[:, head]
    k = unit(proj["k"].view(n, Hk, D))[:, head]
    v = proj["v"].view(n, H, Dv)
    beta = 1 / (1 + torch.exp(-(h @ w[p + "b"].T)))
    o, _ = delta_rule(q, k, v, beta, channel_decay(w, p, H, D, h))
    gate = 1 / (1 + torch.exp(-((h @ w[p + "g1"].T) @ w[p + "g2"].T)))
    o = rms_normalise(o, eps) * w[p + "norm"] * gate.view(n, H, Dv)
    return o.reshape(n, H * Dv) @ w[p + "o"].T


def gated_mlp(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def hyper_in(streams, w_in):
    return sum(w_in[s] * streams[s] for s in range(len(streams)))


def hyper_out(streams, mix, out, y):
    n = len(streams)
    return [sum(mix[s, t] * streams[s] for s in range(n)) + out[t] * y for t in range(n)]


def layer_order(cfg):
    """Layer index of every run, the looped stretch repeated."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


MIXERS = {"latent_attention": latent_attention, "channel_delta": channel_delta}


def forward(cfg, weights, tokens, dtype=torch.float64, residuals=None):
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    xs = [x.clone() for _ in range(cfg["streams"])]
    for i in layer_order(cfg):
        L, l = cfg["layers"][i], f"l{i}."
        subs = [(1, lambda h: MIXERS[L["type"]](w, l + "mix.", L["mixer"], h, eps))]
        if L["mlp"] is not None:
            subs.append((2, lambda h: gated_mlp(w, l + "mlp.", h)))
        for q, f in subs:
            hc = f"{l}hc{q}."
            h = layer_norm(hyper_in(xs, w[hc + "in"]), w[f"{l}norm{q}"], w[f"{l}norm{q}.b"], eps)
            xs = hyper_out(xs, w[hc + "mix"], w[hc + "out"], f(h))
        if residuals is not None:
            residuals.append(sum(xs))
    h = layer_norm(sum(xs), w["final.norm"], w["final.norm.b"], eps)
    return h @ w["embed"].T


def random_weights(cfg, seed=0, a_rank=12, g_rank=20, dtype=torch.float32):
    """Seeded weights with every tensor of ``cfg``, scaled so that each mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)

    def lin(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * s * i ** -0.5

    def near(n, c, s):
        return c + s * torch.randn(n, generator=g)
    E, S = cfg["width"], cfg["streams"]
    w = {"embed": torch.randn(cfg["vocab"], E, generator=g) * E ** -0.5, "final.norm": near(E, 1, 0.1), "final.norm.b": near(E, 0, 0.1)}
    for i, L in enumerate(cfg["layers"]):
        l, m = f"l{i}.", L["mixer"]
        p = l + "mix."
        for q in ((1, 2) if L["mlp"] is not None else (1,)):
            w[f"{l}norm{q}"], w[f"{l}norm{q}.b"] = near(E, 1, 0.1), near(E, 0, 0.1)
            w[f"{l}hc{q}.in"], w[f"{l}hc{q}.out"] = near(S, 1 / S, 0.2), near(S, 1, 0.3)
            w[f"{l}hc{q}.mix"] = torch.eye(S) + 0.2 * torch.randn(S, S, generator=g)
        if L["type"] == "latent_attention":
            H, D, Dv, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
            w[p + "q"], w[p + "dkv"], w[p + "dkv.norm"] = lin(H * D, E, 1.3), lin(R, E), near(R, 1, 0.1)
            w[p + "uk"], w[p + "uv"], w[p + "o"] = lin(H * D, R, 1.3), lin(H * Dv, R), lin(E, H * Dv)
        else:
            H, Hk, D, Dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, ch in (("q", Hk * D), ("k", Hk * D), ("v", H * Dv)):
                w[p + n], w[f"{p}{n}.conv"] = lin(ch, E), 0.5 * torch.randn(ch, K, generator=g)
            w[p + "b"], w[p + "A_log"], w[p + "dt_bias"] = lin(H, E), near(H, -1, 0.7), near(H * D, -2, 1.0)
            w[p + "a1"], w[p + "a2"], w[p + "g1"], w[p + "g2"] = lin(a_rank, E), lin(H * D, a_rank), lin(g_rank, E), lin(H * Dv, g_rank)
            w[p + "norm"], w[p + "o"] = near(Dv, 1, 0.1), lin(E, H * Dv)
        if L["mlp"] is not None:
            F = L["mlp"]["ff"]
            w[l + "mlp.gate"], w[l + "mlp.up"], w[l + "mlp.down"] = lin(F, E), lin(F, E), lin(E, F)
    return {n: t.to(torch.bfloat16).to(dtype) for n, t in w.items()}
