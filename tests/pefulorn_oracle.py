"""Plain, slow reference of the Pefulorn design: one function per mechanism, no batching, no cache, no kernels.

``forward`` runs one whole sequence and returns its logits; ``layers_out`` collects the residual after every layer run.
Weights are a dict of float tensors under the checkpoint's tensor names.  The arithmetic type is that of the weights
(float64 in the tests), and nothing is imported from the package.
"""
import torch
import torch.nn.functional as F


def rms(x, eps):
    """Rows divided by the square root of (mean square + eps)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_one_plus(x, w, eps):
    return rms(x, eps) * (1 + w)


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh((2 / torch.pi) ** 0.5 * (x + 0.044715 * x ** 3)))


def previous(h):
    """Row t - 1 for row t; zeros before the first row."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


# ------------------------------------------------------------------ delta rule with a decay per key channel
def causal_conv(x, w):
    """``x`` [T, C], ``w`` [C, taps]: the last tap multiplies the row itself."""
    taps, out = w.shape[1], torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        out[back:] += x[: len(x) - back] * w[:, j] if back < len(x) else 0
    return out


def channel_decay(z, a_log, dt_bias, heads):
    """``z`` [T, heads * dim] -> decay factors [T, heads, dim]."""
    z = (z + dt_bias).reshape(len(z), heads, -1)
    return torch.exp(-torch.exp(a_log)[:, None] * F.softplus(z, threshold=1e9))


def delta_scan(q, k, v, g, beta, state=None):
    """``q``, ``k``, ``g`` [T, H, a], ``v`` [T, H, b], ``beta`` [T, H] -> ([T, H, b], state [H, a, b])."""
    t, heads, a = q.shape
    s = torch.zeros(heads, a, v.shape[-1]).to(q) if state is None else state
    out = []
    for j in range(t):
        s = g[j][:, :, None] * s
        u = beta[j][:, None] * (v[j] - torch.einsum("hab,ha->hb", s, k[j]))
        s = s + k[j][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hab,ha->hb", s, q[j]))
    return torch.stack(out), s


def channel_delta(w, p, m, eps, h):
    t, heads, kv, dim, vdim = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q, k = (unit(x.reshape(t, kv, dim)).repeat_interleave(heads // kv, dim=1) for x in (q, k))
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = channel_decay(h @ w[p + "a1"].T @ w[p + "a2"].T, w[p + "A_log"], w[p + "dt_bias"], heads)
    o, _ = delta_scan(q * dim ** -0.5, k, v.reshape(t, heads, vdim), g, beta)
    o = rms(o, eps) * w[p + "norm"]
    return (o.reshape(t, -1) * torch.sigmoid(h @ w[p + "g1"].T @ w[p + "g2"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------ attention with a logarithmic distance bias
def temperature(pos, coef, every):
    return 1 + coef * torch.log(torch.div(pos + 1, every, rounding_mode="floor").double() + 1)


def log_bias(dist, r1, r2):
    """[H, ...]: what a score loses at a distance."""
    return r1.reshape(-1, *[1] * dist.dim()) * torch.log(1 + r2.reshape(-1, *[1] * dist.dim()) * dist)


def log_bias_attention(q, k, v, qpos, kpos, scale, r1, r2):
    """``q`` [Tq, H, a], ``k`` [Tk, G, a], ``v`` [Tk, G, b] -> [Tq, H, b]."""
    heads, groups = q.shape[1], k.shape[1]
    k, v = (x.repeat_interleave(heads // groups, dim=1) for x in (k, v))
    dist = qpos[:, None] - kpos[None, :]
    s = torch.einsum("qha,kha->hqk", q, k) * scale - log_bias(dist.clamp(min=0).to(q), r1, r2)
    return torch.einsum("hqk,khb->qhb", torch.softmax(s.masked_fill((dist < 0)[None], float("-inf")), dim=-1), v)


def attention(w, p, m, eps, h):
    """Concatenated heads, before the output projection."""
    t, pos = len(h), torch.arange(len(h))
    q, k, v = ((h @ w[p + n].T + w[p + n + ".b"]).reshape(t, c, -1) for n, c in (("q", m["heads"]), ("k", m["kv_heads"]), ("v", m["kv_heads"])))
    q, k, v = rms(q, eps) * w[p + "q.norm"], rms(k, eps) * w[p + "k.norm"], rms(v, eps)
    if m.get("q_temp"):
        q = q * temperature(pos, m["q_temp"]["coef"], m["q_temp"]["every"]).to(q)[:, None, None]
    return log_bias_attention(q, k, v, pos, pos, m["scale"], w[p + "r1"], w[p + "r2"]).reshape(t, -1)


# ------------------------------------------------------------------ minGRU
def min_gru_scan(z, u, state=None):
    """Pre-activations [T, C] of the gate and the candidate -> ([T, C], state)."""
    s = torch.zeros_like(z[0]) if state is None else state
    z, c, out = torch.sigmoid(z), torch.where(u >= 0, u + 0.5, torch.sigmoid(u)), []
    for j in range(len(z)):
        s = (1 - z[j]) * s + z[j] * c[j]
        out.append(s)
    return torch.stack(out), s


def min_gru(w, p, h):
    s, _ = min_gru_scan(h @ w[p + "z"].T + w[p + "z.b"], h @ w[p + "x"].T + w[p + "x.b"])
    return s * silu(h @ w[p + "g"].T)


def parallel(w, p, m, eps, h):
    return m["left_scale"] * (attention(w, p + "left.", m["left"], eps, h) @ w[p + "left.o"].T) + \
        m["right_scale"] * (min_gru(w, p + "right.", h) @ w[p + "right.o"].T)


# ------------------------------------------------------------------ time mixing
def wkv_scan(r, k, v, g, u, state=None):
    """``r``, ``k``, ``g`` [T, H, a], ``v`` [T, H, b], ``u`` [H, a] -> ([T, H, b], state [H, a, b])."""
    s = torch.zeros(*k.shape[1:], v.shape[-1]).to(k) if state is None else state
    out = []
    for j in range(len(r)):
        kv = k[j][:, :, None] * v[j][:, None, :]
        out.append(torch.einsum("hab,ha->hb", s + u[:, :, None] * kv, r[j]))
        s = g[j][:, :, None] * s + kv
    return torch.stack(out), s


def wkv(w, p, m, eps, h):
    t, before = len(h), previous(h)
    mix = {n: h + (before - h) * w[p + "mu." + n] for n in "rkvgw"}
    r, k, v = ((mix[n] @ w[p + n].T).reshape(t, m["heads"], m["dim"]) for n in "rkv")
    g = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).reshape(r.shape)
    o, _ = wkv_scan(r, k, v, g, w[p + "u"])
    return (rms(o, eps).reshape(t, -1) * w[p + "norm"] * silu(mix["g"] @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------ the rest
def dense(w, p, h):
    return (gelu_tanh(h @ w[p + "gate"].T + w[p + "gate.b"]) * (h @ w[p + "up"].T + w[p + "up.b"])) @ w[p + "down"].T + w[p + "down.b"]


MIXERS = {"channel_delta": channel_delta, "parallel": parallel, "wkv": wkv}


def order_of(cfg):
    """(layer, pass that starts before it or None) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def forward(w, cfg, tokens, layers_out=None):
    eps = cfg["norm"]["eps"]
    x0 = x = w["embed"][torch.as_tensor(tokens)]
    for i, begins in order_of(cfg):
        if begins is not None:
            x = x + (x0 if begins else 0) + w["loop.step"][begins]
        layer, p = cfg["layers"][i], f"l{i}."
        x = x + MIXERS[layer["type"]](w, p + "mix.", layer["mixer"], eps, norm_one_plus(x, w[p + "norm1"], eps))
        if layer["mlp"] is not None:
            x = x + dense(w, p + "mlp.", norm_one_plus(x, w[p + "norm2"], eps))
        if layers_out is not None:
            layers_out.append(x)
    return norm_one_plus(x, w["final.norm"], eps) @ w["head"].T
