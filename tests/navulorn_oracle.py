"""Plain definition of the Navulorn decoder, one function per mechanism, float64, whole sequences, no cache.  Shares nothing with the
engine: tests compare the engine (loader, caches, state lines, ragged batches, kernels) against these functions."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def bigram_rows(tokens, b):
    """Row of the bigram table for every token: the pair's hash, or the row behind the buckets for the first token."""
    rows = [b["buckets"]]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * b["mul_prev"] + int(cur) * b["mul_cur"]) % b["buckets"])
    return rows[:len(tokens)]


def embedding(tokens, w, e):
    x = w["embed"][torch.as_tensor(tokens)] * e.get("scale", 1.0)
    if e.get("bigram"):
        x = x + w["bigram"][torch.as_tensor(bigram_rows(list(tokens), e["bigram"]))]
    return x


def frequencies(rot):
    """f_i of the rotary angles; with ``scaling``: long wavelengths slowed down, a linear blend between the two borders."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wave = 2 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate(x, rot, interleaved):
    """x [T, ..., C]: the first ``dims`` of C are rotated by position; pairs (2i, 2i + 1) or (i, i + dims / 2)."""
    T, dims = x.shape[0], rot["dims"]
    a = torch.arange(T, dtype=torch.float64).unsqueeze(1) * frequencies(rot)
    a = a.view(T, *[1] * (x.dim() - 2), dims // 2)
    y = x.clone()
    at = (slice(0, dims, 2), slice(1, dims, 2)) if interleaved else (slice(0, dims // 2), slice(dims // 2, dims))
    u, v = x[..., at[0]], x[..., at[1]]
    y[..., at[0]] = u * torch.cos(a) - v * torch.sin(a)
    y[..., at[1]] = v * torch.cos(a) + u * torch.sin(a)
    return y


def visible(T, mask):
    i, j = torch.arange(T).view(T, 1), torch.arange(T).view(1, T)
    see = j <= i
    if mask and mask.get("size"):
        see = see & (i - j < mask["size"])
    return see


def softmax_rows(s, see):
    s = s.masked_fill(~see, float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def attention(h, w, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, d)
    k = (rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, d)
    v = (h @ w[p + "v"].T).view(T, G, dv)
    if m.get("rot"):
        q, k = rotate(q, m["rot"], False), rotate(k, m["rot"], False)
    see = visible(T, m.get("mask"))
    gate = torch.sigmoid(h @ w[p + "g"].T)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = gate[:, a:a + 1] * (softmax_rows(q[:, a] @ k[:, g].T * m["scale"], see) @ v[:, g])
    return out.reshape(T, H * dv) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps):
    T, H, d, r, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    kv = h @ w[p + "dkv"].T
    c = rms(kv[:, :R], eps) * w[p + "dkv.norm"]
    k_rot = rotate(kv[:, R:], m["rot"], True)
    q_rot = rotate(q[..., d:], m["rot"], True)
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    see = visible(T, m.get("mask"))
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        s = (q[:, a, :d] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]
        out[:, a] = softmax_rows(s, see) @ v[:, a]
    return out.reshape(T, H * dv) @ w[p + "o"].T


def mlstm_gates(h, w, p, cap):
    """(log input gate, log forget gate), each [T, heads]."""
    soft = lambda n: cap * torch.tanh((h @ w[p + n].T + w[p + n + ".b"]) / cap)          # noqa: E731
    return soft("i"), torch.nn.functional.logsigmoid(soft("f"))


def mlstm_states(q, k, v, i, f):
    """The recurrence over [T, H, ...] rows, step by step; -> outputs [T, H, Dv]."""
    T, H, D = q.shape
    Dv = v.shape[-1]
    S, n, mx = torch.zeros(H, D, Dv, dtype=q.dtype), torch.zeros(H, D, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    out = torch.zeros(T, H, Dv, dtype=q.dtype)
    for t in range(T):
        new = torch.maximum(f[t] + mx, i[t])
        fade, put = torch.exp(f[t] + mx - new), torch.exp(i[t] - new)
        mx = new
        S = fade.view(H, 1, 1) * S + put.view(H, 1, 1) * k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        n = fade.view(H, 1) * n + put.view(H, 1) * k[t]
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-mx)) + 1e-6
        out[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den.unsqueeze(-1)
    return out


def mlstm(h, w, p, m, eps):
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k, v = (h @ w[p + "k"].T).view(T, H, D), (h @ w[p + "v"].T).view(T, H, Dv)
    o = mlstm_states(q, k, v, *mlstm_gates(h, w, p, m["gate_cap"]))
    o = rms(o, eps).reshape(T, H * Dv) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def dense_ff(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top):
    """-> (weights, ids), each [T, top]: the largest logits, softmax over them alone."""
    best, idx = z.sort(-1, descending=True)
    return torch.softmax(best[:, :top], -1), idx[:, :top]


def moe_ff(h, w, p, f):
    wt, idx = route(h @ w[p + "router"].T + w[p + "router.b"], f["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(idx.shape[1]):
            e = f"{p}e{int(idx[t, k])}."
            a = h[t] @ w[e + "gate"].T
            out[t] += wt[t, k] * ((a * torch.sigmoid(a) * (h[t] @ w[e + "up"].T)) @ w[e + "down"].T)
    return out


MIXERS = {"attention": attention, "latent_attention": latent_attention, "mlstm": mlstm}


def forward(cfg, w, tokens, streams=None):
    """Logits [T, vocab] (float64) of one whole sequence; ``streams`` collects the residual stream after every layer."""
    w = {k: v.double() for k, v in w.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = embedding(tokens, w, cfg.get("embedding") or {})
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = rms(alpha * x + MIXERS[spec["type"]](x, w, p + "mix.", spec["mixer"], eps), eps) * w[p + "norm1"]
        f = spec.get("mlp")
        if f is not None:
            y = dense_ff(x, w, p + "mlp.") if f["kind"] == "dense" else moe_ff(x, w, p + "mlp.", f)
            x = rms(alpha * x + y, eps) * w[p + "norm2"]
        if streams is not None:
            streams.append(x.clone())
    z = (rms(x, eps) * w["final.norm"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z
