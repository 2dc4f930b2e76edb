"""Plain, slow reference of the Napadra design: one function per mechanism, no batching, no cache, no kernels.

``forward`` runs one whole sequence and returns its logits; ``layers_out`` collects the sum of the residual streams after
every layer.  Weights are a dict of float tensors under the checkpoint's tensor names.  The arithmetic type is that of the
weights (float64 in the tests), and nothing is imported from the package.
"""
import torch


def rms(x, eps):
    """Rows divided by the square root of (mean square + eps)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def sinusoid(pos, width):
    """Position vectors [T, width]: sine and cosine of the same angle in turn."""
    out = torch.zeros(len(pos), width, dtype=torch.float64)
    for c in range(width):
        a = pos.double() * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.sin(a) if c % 2 == 0 else torch.cos(a)
    return out


def previous(h):
    """Row t - 1 for row t; zeros before the first row."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def token_shift(h, mu):
    return h + (previous(h) - h) * mu


def streams_in(x, a):
    """``x`` [S, T, W], ``a`` [S]: what a sublayer reads."""
    return torch.einsum("s,stw->tw", a, x)


def streams_out(x, mix, out, y, mult):
    """New streams from the old ones (``mix`` [from, to]) and the sublayer's result."""
    return torch.einsum("sr,stw->rtw", mix, x) + mult * out[:, None, None] * y[None]


def alibi_slopes(heads):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float64)


def same_chunk(qpos, kpos, size):
    """Key ``j`` is seen from ``i`` when it is not later and in the same chunk (``size`` None: one chunk)."""
    ok = kpos[None, :] <= qpos[:, None]
    return ok & (qpos[:, None] // size == kpos[None, :] // size) if size else ok


def sink_attention(q, k, v, qpos, kpos, size, scale, sink):
    """``q`` [Tq, H, a], ``k`` [Tk, G, a], ``v`` [Tk, G, b] -> [Tq, H, b]."""
    heads, groups = q.shape[1], k.shape[1]
    k, v = (t.repeat_interleave(heads // groups, dim=1) for t in (k, v))
    s = torch.einsum("qha,kha->hqk", q, k) * scale
    s = s - alibi_slopes(heads).to(s)[:, None, None] * (qpos[:, None] - kpos[None, :]).to(s)
    s = s.masked_fill(~same_chunk(qpos, kpos, size)[None], float("-inf"))
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    p = e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))
    return torch.einsum("hqk,khb->qhb", p, v)


def attention(w, p, src, m, h, kept):
    """``p``: tensor prefix of the layer's mixer; ``src``: layer whose keys and values it reads (``kept``: by layer)."""
    t = len(h)
    if src not in kept:
        kept[src] = ((h @ w[p + "k"].T).reshape(t, m["kv_heads"], m["dim"]),
                     (h @ w[p + "v"].T).reshape(t, m["kv_heads"], m["vdim"]))
    k, v = kept[src]
    q = (h @ w[p + "q"].T).reshape(t, m["heads"], m["dim"])
    pos = torch.arange(t)
    o = sink_attention(q, k, v, pos, pos, (m.get("mask") or {}).get("size"), m["scale"], w[p + "sink"])
    return o.reshape(t, -1) @ w[p + "o"].T


def mlstm_gates(zi, zf, cap):
    """(log input gate, log forget gate) from the gates' pre-activations."""
    return cap * torch.tanh(zi / cap), torch.nn.functional.logsigmoid(cap * torch.tanh(zf / cap))


def mlstm_scan(q, k, v, i, f, state=None):
    """``q``, ``k`` [T, H, a] (``q`` scaled), ``v`` [T, H, b], log gates [T, H] -> ([T, H, b], state)."""
    t, heads, a = q.shape
    if state is None:
        state = (torch.zeros(heads, a, v.shape[-1]).to(q), torch.zeros(heads, a).to(q), torch.zeros(heads).to(q))
    s, n, m = state
    out = []
    for j in range(t):
        new = torch.maximum(f[j] + m, i[j])
        keep, add = torch.exp(f[j] + m - new), torch.exp(i[j] - new)
        m = new
        s = keep[:, None, None] * s + add[:, None, None] * k[j][:, :, None] * v[j][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[j]
        den = torch.maximum((n * q[j]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hab,ha->hb", s, q[j]) / den[:, None])
    return torch.stack(out), (s, n, m)


def mlstm(w, p, m, eps, h):
    t, heads = len(h), m["heads"]
    q = (h @ w[p + "q"].T).reshape(t, heads, m["dim"]) * m["dim"] ** -0.5
    k = (h @ w[p + "k"].T).reshape(t, heads, m["dim"])
    v = (h @ w[p + "v"].T).reshape(t, heads, m["vdim"])
    i, f = mlstm_gates(h @ w[p + "i"].T + w[p + "i.b"], h @ w[p + "f"].T + w[p + "f.b"], m["gate_cap"])
    o, _ = mlstm_scan(q, k, v, i, f)
    return (rms(o, eps).reshape(t, -1) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def dense(w, p, f, h):
    return clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, f["limit"]) @ w[p + "down"].T


def forward(w, cfg, tokens, layers_out=None):
    eps, width, mult = cfg["norm"]["eps"], cfg["width"], cfg["residual_mult"]
    tokens = torch.as_tensor(tokens)
    x0 = w["embed"][tokens] + sinusoid(torch.arange(len(tokens)), width).to(w["embed"])
    x = x0[None].repeat(cfg["streams"], 1, 1)
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms(streams_in(x, w[p + "hc1.in"]), eps) * w[p + "norm1"]
        h = token_shift(h, w[p + "shift"])
        if layer["type"] == "mlstm":
            y = mlstm(w, p + "mix.", m, eps, h)
        else:
            y = attention(w, p + "mix.", m.get("kv_from", i), m, h, kept)
        x = streams_out(x, w[p + "hc1.mix"], w[p + "hc1.out"], y * w[p + "ls1"], mult)
        if layer["mlp"] is not None:
            h = rms(streams_in(x, w[p + "hc2.in"]), eps) * w[p + "norm2"]
            y = dense(w, p + "mlp.", layer["mlp"], h)
            x = streams_out(x, w[p + "hc2.mix"], w[p + "hc2.out"], y * w[p + "ls2"], mult)
        if layers_out is not None:
            layers_out.append(x.sum(0))
    return rms(x.sum(0), eps) * w["final.norm"] @ w["head"].T
