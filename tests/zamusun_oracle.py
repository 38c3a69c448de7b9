"""Plain, slow restatement of the Zamusun design for the tests: one function per mechanism, straight from the equations, in
whatever floating type the tensors have (the tests use float64). It shares no code with the package.

Notation: ``t`` token rows, ``h`` heads, all sequences start at position 0. ``mix`` and ``mlp`` are the plain dictionaries of
a layer's entry in config.json, ``w`` maps tensor names to tensors.
"""

import math

import torch


def rms(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def linear(x, w, name):
    y = x @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


def query_temperature(positions, coef, every):
    """1 + coef ln(floor((p + 1) / every) + 1)"""
    return 1 + coef * torch.log(torch.div(positions + 1, every, rounding_mode="floor").double() + 1)


def softmax_with_sink(scores, sink):
    """scores [h, t, t] (-inf where hidden), sink [h]: weights whose denominator also has exp(sink)."""
    top = torch.maximum(scores.amax(-1), sink[:, None])
    e = torch.exp(scores - top[..., None])
    return e / (e.sum(-1) + torch.exp(sink[:, None] - top))[..., None]


def attention(h, w, name, mix, eps):
    """Grouped heads whose values are their keys."""
    t, H, G, D = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"]
    q = linear(h, w, name + ".q").view(t, H, D)
    k = linear(h, w, name + ".k").view(t, G, D)
    positions = torch.arange(t)
    q = q * query_temperature(positions, mix["q_temp"]["coef"], mix["q_temp"]["every"]).to(h.dtype)[:, None, None]
    k = k.repeat_interleave(H // G, 1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * mix["scale"]
    scores = scores.masked_fill(positions[None, :] > positions[:, None], -math.inf)
    p = softmax_with_sink(scores, w[name + ".sink"])
    o = torch.einsum("hij,jhd->ihd", p, k).reshape(t, H * D)
    return linear(o * torch.sigmoid(linear(h, w, name + ".g")), w, name + ".o")


def lightning_scan(q, k, v, decay):
    """S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t;  q, k [t, h, d], v [t, h, e]."""
    t, H, D = q.shape
    S = q.new_zeros(H, D, v.shape[-1])
    g = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    out = []
    for i in range(t):
        S = g * S + k[i][:, :, None] * v[i][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[i]))
    return torch.stack(out)


def silu(z):
    return z * torch.sigmoid(z)


def lightning(h, w, name, mix, eps):
    t, H = h.shape[0], mix["heads"]
    q = silu(linear(h, w, name + ".q")).view(t, H, mix["dim"])
    k = silu(linear(h, w, name + ".k")).view(t, H, mix["dim"])
    v = silu(linear(h, w, name + ".v")).view(t, H, mix["vdim"])
    o = lightning_scan(q, k, v, mix["decay"]).reshape(t, H * mix["vdim"])
    o = rms(o, eps) * w[name + ".norm"]
    return linear(o * torch.sigmoid(linear(h, w, name + ".g")), w, name + ".o")


def mlstm_gates(h, w, name, cap):
    """Logarithms of the input gate and of the forget gate, [t, h]."""
    i = cap * torch.tanh(linear(h, w, name + ".i") / cap)
    f = cap * torch.tanh(linear(h, w, name + ".f") / cap)
    return i, -torch.log1p(torch.exp(-f))


def mlstm_scan(q, k, v, i, f):
    """Matrix memory with a running maximum m that starts at 0;  q (scaled), k [t, h, d], v [t, h, e], i, f [t, h]."""
    t, H, D = q.shape
    S, n, m = q.new_zeros(H, D, v.shape[-1]), q.new_zeros(H, D), q.new_zeros(H)
    out = []
    for s in range(t):
        new = torch.maximum(f[s] + m, i[s])
        keep, write = torch.exp(f[s] + m - new), torch.exp(i[s] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[s][:, :, None] * v[s][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[s]
        m = new
        norm = torch.maximum((n * q[s]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[s]) / norm[:, None])
    return torch.stack(out)


def mlstm(h, w, name, mix, eps):
    t, H, D = h.shape[0], mix["heads"], mix["dim"]
    q = linear(h, w, name + ".q").view(t, H, D) * D ** -0.5
    k = linear(h, w, name + ".k").view(t, H, D)
    v = linear(h, w, name + ".v").view(t, H, mix["vdim"])
    i, f = mlstm_gates(h, w, name, mix["gate_cap"])
    o = rms(mlstm_scan(q, k, v, i, f), eps).reshape(t, H * mix["vdim"])
    return linear(o * w[name + ".norm"] * torch.sigmoid(linear(h, w, name + ".g")), w, name + ".o")


MIXERS = {"attention": attention, "lightning": lightning, "mlstm": mlstm}


def expert(h, w, name, limit):
    g = torch.clamp(h @ w[name + ".gate"].T, max=limit)
    u = torch.clamp(h @ w[name + ".up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[name + ".down"].T


def route(z, top):
    """Chosen experts and their weights [t, top]: softmax over all, the largest scores, divided by their sum."""
    s = torch.softmax(z, -1)
    best = torch.sort(s, dim=-1, descending=True, stable=True).indices[:, :top]
    p = torch.gather(s, -1, best)
    return best, p / (p.sum(-1, keepdim=True) + 1e-20)


def experts(h, w, name, mlp):
    best, p = route(h @ w[name + ".router"].T, mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, j = (best == e).nonzero(as_tuple=True)
        out[t] += p[t, j, None] * expert(h[t], w, f"{name}.e{e}", mlp["expert"]["limit"])
    return out


def layer_order(config):
    """(index, first layer of a pass) for every layer run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for i in range(a, b)] * loop["times"] + [(i, False) for i in range(b, n)]


def forward(tokens, w, config, trace=None):
    """Logits [t, vocab] of one sequence; ``trace`` (a list) receives the residual stream after every layer run."""
    eps = config["norm"]["eps"]
    x = x0 = w["embed"][torch.as_tensor(tokens)]
    for i, first in layer_order(config):
        if first:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T
        n, spec = f"l{i}", config["layers"][i]
        h = rms(x, eps) * (1 + w[n + ".norm1"])
        y = MIXERS[spec["type"]](h, w, n + ".mix", spec["mixer"], eps)
        if spec["mlp"] is not None:
            y = y + experts(h, w, n + ".mlp", spec["mlp"])
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, eps) * (1 + w["final.norm"])) @ w["embed"].T
