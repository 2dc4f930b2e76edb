"""Plain, slow reference of the Mumusun design: one function per mechanism, no batching, no cache, no kernels.

``forward`` runs one whole sequence and returns its logits; ``layers_out`` collects the residual stream after every
layer.  Weights are a dict of float tensors under the checkpoint's tensor names.  The arithmetic type is that of the
weights (float64 in the tests), and nothing is imported from the package.
"""
import torch


def layer_norm(x, w, eps):
    """Deviation from the mean over the square root of (mean squared deviation + eps), times a weight; no bias."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def rotate(x, pos, dims, base):
    """Rotate-half positions on the first ``dims`` of the last axis; ``x`` [T, ..., n], ``pos`` [T]."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = (pos.double()[:, None] * f).reshape([len(pos)] + [1] * (x.dim() - 2) + [half])
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], dim=-1)


def visible(qpos, kpos, window):
    """Key ``j`` is seen from position ``i`` when ``0 <= i - j < window`` (``window`` None: every earlier key)."""
    d = qpos[:, None] - kpos[None, :]
    return (d >= 0) & (d < window) if window else d >= 0


def softmax_attention(q, k, v, mask, scale):
    """``q`` [Tq, H, a], ``k`` [Tk, H, a], ``v`` [Tk, H, b] -> [Tq, H, b]."""
    s = torch.einsum("qha,kha->hqk", q, k) * scale
    s = s.masked_fill(~mask[None], float("-inf"))
    return torch.einsum("hqk,khb->qhb", torch.softmax(s, dim=-1), v)


def latent_attention(w, p, m, eps, h, pos):
    """The whole mixer over one sequence; ``p`` the tensor prefix, ``m`` the mixer's configuration."""
    t, heads, dim, rot, vdim, rank = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).reshape(t, heads, dim + rot)
    kv = h @ w[p + "dkv"].T
    c = rms_norm(kv[:, :rank], w[p + "dkv.norm"], eps)
    rdims, base = m["rot"]["dims"], m["rot"]["base"]
    kr = rotate(kv[:, rank:], pos, rdims, base)
    qr = rotate(q[..., dim:], pos, rdims, base)
    k = torch.cat([(c @ w[p + "uk"].T).reshape(t, heads, dim), kr[:, None, :].expand(t, heads, rot)], dim=-1)
    v = (c @ w[p + "uv"].T).reshape(t, heads, vdim)
    window = (m.get("mask") or {}).get("size")
    o = softmax_attention(torch.cat([q[..., :dim], qr], dim=-1), k, v, visible(pos, pos, window), m["scale"])
    return o.reshape(t, heads * vdim) @ w[p + "o"].T


def route(z, r):
    """Chosen experts of one token (list of (expert, weight)) from its router logits ``z``."""
    s = torch.sigmoid(z)
    n, top = r["experts"], r["top"]
    allowed = set(range(n))
    g = r.get("groups")
    if g:
        size = n // g["count"]
        score = [float(sum(sorted((float(x) for x in s[i * size:(i + 1) * size]), reverse=True)[:2])) for i in range(g["count"])]
        best = sorted(range(g["count"]), key=lambda i: (-score[i], i))[: g["keep"]]
        allowed = {i * size + j for i in best for j in range(size)}
    order = sorted(allowed, key=lambda e: (-float(s[e]), e))[:top]
    return [(e, s[e]) for e in order]


def silu(z):
    return z * torch.sigmoid(z)


def expert(w, p, x):
    return w[p + "down"] @ (silu(w[p + "gate"] @ x) * (w[p + "up"] @ x))


def moe(w, p, cfg, h):
    z = h @ w[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(len(h)):
        for e, s in route(z[t], cfg["router"]):
            out[t] += s * expert(w, f"{p}e{e}.", h[t])
    return out


def forward(w, cfg, tokens, layers_out=None):
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = w["embed"][torch.as_tensor(tokens)].clone()
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + layer_norm(latent_attention(w, p + "mix.", layer["mixer"], eps, x, pos), w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + layer_norm(moe(w, p + "mlp.", layer["mlp"], x), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T
