"""Plain float64 definition of the Balivik decoder, one function per mechanism, whole sequences only (no cache, no state handed between
calls, no batches).  The tests compare the engine with this file; nothing here is shared with the product path."""
import math

import torch

F64 = torch.float64


def rms_norm(x, eps, w=None):
    """x over its last axis, divided by the root of (its mean square + eps), times w (a vector or one number)."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(x):
    return x * torch.sigmoid(x)


def causal_conv(x, w):
    """x [T, C], w [C, K]: y[t] = sum over d < K of w[:, K - 1 - d] * x[t - d]; rows before the sequence count as zero."""
    T, K = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for d in range(K):
        if d < T:
            y[d:] += w[:, K - 1 - d] * x[:T - d]
    return y


def rotate(x, rot, first_position=0):
    """x [T, H, D]: channels i and i + dims / 2 (i < dims / 2) form a point that turns by position * base^(-2 i / dims); the channels from
    ``dims`` on are copied."""
    d = int((rot or {}).get("dims") or 0)
    if not d:
        return x
    f = torch.tensor([rot["base"] ** (-2.0 * i / d) for i in range(d // 2)], dtype=F64)
    a = torch.arange(first_position, first_position + x.shape[0], dtype=F64)[:, None] * f[None]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :d // 2], x[..., d // 2:d]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., d:]], -1)


def causal_attention(q, k, v, scale):
    """One head: q, k [T, D], v [T, Dv]; row i weighs rows 0 .. i."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], -float("inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return (e / e.sum(-1, keepdim=True)) @ v


def lambda_of(lq1, lk1, lq2, lk2, diff):
    return float(torch.exp((lq1.double() * lk1.double()).sum()) - torch.exp((lq2.double() * lk2.double()).sum()) + diff)


def differential_attention(q, k, v, scale, lam, diff, eps):
    """q [T, H, 2, D], k [T, G, 2, D], v [T, G, Dv]: two softmax maps per head over the same values; the second, times lam, is taken off
    the first, and what is left is normalised over the value channels and multiplied by 1 - diff.  [T, H, Dv]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        a1, a2 = (causal_attention(q[:, h, m], k[:, g, m], v[:, g], scale) for m in (0, 1))
        out[:, h] = rms_norm(a1 - lam * a2, eps) * (1.0 - diff)
    return out


def decayed_outer_products(q, k, v, decay):
    """q, k [T, H, D], v [T, H, Dv], decay [H]: what a head reads at step t is sum over s <= t of decay^(t - s) (q_t . k_s) v_s."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64)
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def channel_delta_rule(q, k, v, beta, decay):
    """q, k, decay [T, H, D], v [T, H, Dv], beta [T, H].  Per step every row of the state shrinks by its own key channel's decay; the state
    is then corrected along k towards v with strength beta, and read at q after the correction."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64)
    out = []
    for t in range(T):
        S = decay[t][:, :, None] * S
        miss = v[t] - (S * k[t][:, :, None]).sum(1)
        S = S + k[t][:, :, None] * (beta[t][:, None] * miss)[:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def unit(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def mixer_attention(h, m, w, p, eps):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rotate((h @ w[p + "q"].T).view(T, H * 2, D), m.get("rot")).view(T, H, 2, D)
    k = rotate((h @ w[p + "k"].T).view(T, G * 2, D), m.get("rot")).view(T, G, 2, D)
    v = (h @ w[p + "v"].T).view(T, G, m["vdim"])
    lam = lambda_of(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    return differential_attention(q, k, v, m["scale"], lam, m["diff"], eps).reshape(T, -1) @ w[p + "o"].T


def mixer_lightning(h, m, w, p, eps):
    T, H = h.shape[0], m["heads"]
    q, k, v = (silu(h @ w[p + n].T).view(T, H, -1) for n in ("q", "k", "v"))
    o = decayed_outer_products(q, k, v, torch.tensor(m["decay"], dtype=F64)).reshape(T, -1)
    return (rms_norm(o, eps, w[p + "norm"]) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mixer_channel_delta(h, m, w, p, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = (unit(q.view(T, G, D)) * D ** -0.5).repeat_interleave(H // G, 1)
    k = unit(k.view(T, G, D)).repeat_interleave(H // G, 1)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    a = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    decay = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(a).view(T, H, D))
    o = rms_norm(channel_delta_rule(q, k, v.view(T, H, Dv), beta, decay), eps, w[p + "norm"]).reshape(T, -1)
    return (o * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)) @ w[p + "o"].T


MIXERS = dict(attention=mixer_attention, lightning=mixer_lightning, channel_delta=mixer_channel_delta)


def dense(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def clamped_expert(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def table_moe(h, tokens, f, w, p):
    """Every token's experts stand in its row of the table; all of them count the same."""
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens):
        chosen = w[p + "table"][tok].tolist()
        for e in chosen:
            out[t] += clamped_expert(h[t:t + 1], w, f"{p}e{int(e)}.", f["expert"]["limit"])[0] / len(chosen)
    return out


def mix_streams(x, y, w, p):
    """x [S, T, W]: stream t becomes sum_s mix[s, t] x_s + out[t] y."""
    return torch.einsum("st,snw->tnw", w[p + "mix"], x) + w[p + "out"][:, None, None] * y[None]


def read_streams(x, w, p):
    return torch.einsum("s,snw->nw", w[p + "in"], x)


def runs_of(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, w, tokens, streams=None):
    """Logits [T, vocab] of one whole sequence; ``streams`` collects the sum of the streams after every layer run."""
    w = {k: v.double() for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)].expand(cfg["streams"], -1, -1)
    for i in runs_of(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        h = rms_norm(read_streams(x, w, p + "hc1."), eps, w[p + "norm1"])
        if p + "canon1" in w:
            h = h + causal_conv(h, w[p + "canon1"])
        x = mix_streams(x, MIXERS[L["type"]](h, L["mixer"], w, p + "mix.", eps), w, p + "hc1.")
        f = L.get("mlp")
        if f is not None:
            h = rms_norm(read_streams(x, w, p + "hc2."), eps, w[p + "norm2"])
            x = mix_streams(x, dense(h, w, p + "mlp.") if f["kind"] == "dense" else table_moe(h, tokens, f, w, p + "mlp."), w, p + "hc2.")
        if streams is not None:
            streams.append(x.sum(0))
    return rms_norm(x.sum(0), eps, w["final.norm"]) @ w["head"].T * cfg["logit_scale"]
