"""Plain, slow restatement of the Sumitar design for the tests: one function per mechanism, straight from the equations, in
whatever floating type the tensors have (the tests use float64). It shares no code with the package.

Notation: ``t`` token rows, ``h`` heads, all sequences start at position 0. ``mix`` and ``mlp`` are the plain dictionaries of
a layer's entry in config.json, ``w`` maps tensor names to tensors.
"""

import math

import torch


def rms(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def linear(x, w, name):
    y = x @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


def heads(x, n):
    return x.view(len(x), n, -1)


def bounded(x, w, name):
    """The norm that computes no statistics."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


# ---- attention
def rotate(x, rot):
    """x [t, h, d]: channels (i, i + n) of the first 2n, turned by position times frequency."""
    n = rot["dims"] // 2
    f = torch.tensor([rot["base"] ** (-2 * i / rot["dims"]) for i in range(n)], dtype=torch.float64)
    a = torch.arange(len(x), dtype=torch.float64)[:, None] * f
    c, s = (g(a).to(x.dtype)[:, None] for g in (torch.cos, torch.sin))
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def seen_window(t, size):
    i, j = torch.arange(t)[:, None], torch.arange(t)[None]
    return (j <= i) & (i - j < size)


def attend(q, k, v, factor, seen):
    """Grouped softmax attention: q [t, H, d], k [t, G, d], v [t, G, e], factor [H] of the scores -> [t, H, e]."""
    n = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(n, 1), v.repeat_interleave(n, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * factor[:, None, None]
    return torch.einsum("hij,jhe->ihe", torch.softmax(s.masked_fill(~seen, -math.inf), -1), v)


def window_attention(h, w, name, mix):
    """Left half of 'parallel': biases, rotation, a temperature per head, sliding window."""
    q = rotate(heads(linear(h, w, name + ".q"), mix["heads"]), mix["rot"])
    k = rotate(heads(linear(h, w, name + ".k"), mix["kv_heads"]), mix["rot"])
    v = heads(linear(h, w, name + ".v"), mix["kv_heads"])
    o = attend(q, k, v, mix["scale"] * w[name + ".temp"], seen_window(len(h), mix["mask"]["size"]))
    return linear(o.flatten(1), w, name + ".o")


# ---- recurrences
def forget_scan(q, f, v):
    """A matrix per head; what a key row forgets is what the token may write there;  q, f [t, h, d], v [t, h, e]."""
    S, out = v.new_zeros(q.shape[1], q.shape[2], v.shape[2]), []
    for i in range(len(q)):
        S = f[i][:, :, None] * S + (1 - f[i])[:, :, None] * v[i][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[i]))
    return torch.stack(out)


def forget_mix(h, w, name, mix, eps):
    """Right half of 'parallel' (HGRN2)."""
    H, low = mix["heads"], w[name + ".lower"]
    f = low + (1 - low) * torch.sigmoid(linear(h, w, name + ".f"))
    o = forget_scan(heads(silu(linear(h, w, name + ".q")), H), heads(f, H), heads(linear(h, w, name + ".v"), H))
    return linear((rms(o, eps) * w[name + ".norm"]).flatten(1), w, name + ".o")


def side_by_side(h, w, name, mix, eps):
    left, right = window_attention(h, w, name + ".left", mix["left"]), forget_mix(h, w, name + ".right", mix["right"], eps)
    return (rms(left, eps) * w[name + ".left.out"] + rms(right, eps) * w[name + ".right.out"]) / 2


def causal_conv(u, taps):
    """Every channel: the value d tokens back weighs with the d-th tap from the end; nothing lies before the first token."""
    y = torch.zeros_like(u)
    for d, tap in enumerate(taps.flip(1).T):
        if d < len(u):
            y[d:] += tap * u[:len(u) - d]
    return y


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def delta_scan(q, k, v, g, beta):
    """A matrix per head that decays by g and is then corrected towards v at k;  q, k [t, h, d], v [t, h, e], g, beta [t, h]."""
    S, out = v.new_zeros(q.shape[1], q.shape[2], v.shape[2]), []
    for i in range(len(q)):
        S = g[i][:, None, None] * S
        u = beta[i][:, None] * (v[i] - torch.einsum("hde,hd->he", S, k[i]))
        S = S + k[i][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[i]))
    return torch.stack(out)


def delta_mix(h, w, name, mix, eps):
    """'delta': short convolutions with SiLU, unit queries and keys shared by groups of heads, gated norm per head."""
    n = mix["heads"] // mix["kv_heads"]
    q, k, v = (silu(causal_conv(linear(h, w, f"{name}.{s}"), w[f"{name}.{s}.conv"])) for s in "qkv")
    q = unit(heads(q, mix["kv_heads"])).repeat_interleave(n, 1) * mix["dim"] ** -0.5
    k = unit(heads(k, mix["kv_heads"])).repeat_interleave(n, 1)
    beta = torch.sigmoid(h @ w[name + ".b"].T)
    g = torch.exp(-torch.exp(w[name + ".A_log"]) * softplus(h @ w[name + ".a"].T + w[name + ".dt_bias"]))
    o = rms(delta_scan(q, k, heads(v, mix["heads"]), g, beta), eps) * w[name + ".norm"]
    return linear(o.flatten(1) * silu(linear(h, w, name + ".g")), w, name + ".o")


MIXERS = {"parallel": side_by_side, "delta": delta_mix}


# ---- feed-forwards
def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense(h, w, name, eps):
    return linear(poly_norm(linear(h, w, name + ".up"), w[name + ".act"], eps), w, name + ".down")


def gated_unit(h, w, name):
    return linear(silu(linear(h, w, name + ".gate")) * linear(h, w, name + ".up"), w, name + ".down")


def route(z, correction, top):
    """Chosen experts by corrected score, and their plain softmax scores [t, top]."""
    s = torch.softmax(z, -1)
    best = torch.sort(s + correction, dim=-1, descending=True, stable=True).indices[:, :top]
    return best, torch.gather(s, -1, best)


def experts(h, w, name, mlp):
    """The choices behind the experts hand the input on; one expert sees every token, through a gate."""
    best, p = route(linear(h, w, name + ".router"), w[name + ".correction"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    n = mlp["router"]["experts"]
    for e in range(n + mlp["router"].get("identity", 0)):
        t, j = (best == e).nonzero(as_tuple=True)
        out[t] += p[t, j, None] * (gated_unit(h[t], w, f"{name}.e{e}") if e < n else h[t])
    if mlp.get("shared"):
        out = out + torch.sigmoid(linear(h, w, name + ".shared.sg")) * gated_unit(h, w, name + ".shared")
    return out


def feed_forward(h, w, name, mlp, eps):
    return dense(h, w, name, eps) if mlp["kind"] == "dense" else experts(h, w, name, mlp)


def forward(tokens, w, config, trace=None):
    """Logits [t, vocab] of one sequence; ``trace`` (a list) receives the residual stream after every layer."""
    eps, x = config["norm"]["eps"], w["embed"][torch.as_tensor(tokens)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        y = MIXERS[layer["type"]](bounded(x, w, p + ".norm1"), w, p + ".mix", layer["mixer"], eps)
        x = x + bounded(y, w, p + ".norm1b")
        if layer["mlp"] is not None:
            x = x + bounded(feed_forward(bounded(x, w, p + ".norm2"), w, p + ".mlp", layer["mlp"], eps), w, p + ".norm2b")
        if trace is not None:
            trace.append(x.clone())
    return bounded(x, w, "final.norm") @ w["embed"].T
