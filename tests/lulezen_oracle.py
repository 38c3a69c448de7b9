"""Plain, slow restatement of the Lulezen design for the tests: one function per mechanism, straight from the
equations, in whatever floating type the tensors have (the tests use float64). It shares no code with the package.

Notation: ``t`` token rows, ``h`` heads, all sequences start at position 0. ``spec`` is the plain dictionary of a
layer's entry in config.json, ``w`` maps tensor names to tensors.
"""

import math

import torch


def rms(v, weight, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * weight


def layer_norm(v, weight, bias, eps):
    centred = v - v.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * weight + bias


def rotate(v, positions, n_dims, base):
    """Rotate pairs (i, i + n_dims/2) of the last axis by position * base^(-2i/n_dims); v is [t, ..., D]."""
    out = v.clone()
    half = n_dims // 2
    for i in range(half):
        angle = positions.to(v.dtype) * base ** (-2.0 * i / n_dims)
        shape = [-1] + [1] * (v.dim() - 2)
        c, s = torch.cos(angle).view(shape), torch.sin(angle).view(shape)
        a, b = v[..., i], v[..., i + half]
        out[..., i] = a * c - b * s
        out[..., i + half] = b * c + a * s
    return out


def visible(n, window):
    """[n, n] boolean: row i sees column j when 0 <= i - j < window."""
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    return (i - j >= 0) & (i - j < window)


def softmax_with_sink(scores, sink):
    """scores [h, t, t] (-inf where hidden), sink [h]: weights whose denominator also has exp(sink)."""
    top = torch.maximum(scores.amax(-1), sink[:, None])
    e = torch.exp(scores - top[..., None])
    return e / (e.sum(-1) + torch.exp(sink[:, None] - top))[..., None]


def latent_attention(x, positions, w, name, mix, eps):
    t, H = x.shape[0], mix["heads"]
    dim, rot, vdim, rank = mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    c_q = rms(x @ w[name + ".dq"].T, w[name + ".dq.norm"], eps)
    q = (c_q @ w[name + ".uq"].T).view(t, H, dim + rot)
    down = x @ w[name + ".dkv"].T
    c = rms(down[:, :rank], w[name + ".dkv.norm"], eps)
    k_rot = rotate(down[:, rank:], positions, mix["rot"]["dims"], mix["rot"]["base"])
    q_rot = rotate(q[..., dim:], positions, mix["rot"]["dims"], mix["rot"]["base"])
    k = (c @ w[name + ".uk"].T).view(t, H, dim)
    v = (c @ w[name + ".uv"].T).view(t, H, vdim)
    scores = (torch.einsum("ihd,jhd->hij", q[..., :dim], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * mix["scale"]
    scores = scores.masked_fill(~visible(t, mix["mask"]["size"])[None], -math.inf)
    p = softmax_with_sink(scores, w[name + ".sink"])
    o = torch.einsum("hij,jhv->ihv", p, v)
    o = o * torch.sigmoid(x @ w[name + ".g"].T)[..., None]
    return o.reshape(t, H * vdim) @ w[name + ".o"].T


def clamped_swiglu(x, w, name, limit):
    g = torch.clamp(x @ w[name + ".gate"].T, max=limit)
    u = torch.clamp(x @ w[name + ".up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[name + ".down"].T


def forward(tokens, w, config, trace=None):
    """Logits [t, vocab] of one sequence; ``trace`` (a list) receives the residual stream after every layer."""
    eps = config["norm"]["eps"]
    positions = torch.arange(len(tokens))
    x = w["embed"][torch.as_tensor(tokens)]
    for i, spec in enumerate(config["layers"]):
        n = f"l{i}"
        y = latent_attention(x, positions, w, n + ".mix", spec["mixer"], eps)
        x = x + layer_norm(y, w[n + ".norm1"], w[n + ".norm1.b"], eps) * w[n + ".ls1"]
        if spec["mlp"] is not None:
            y = clamped_swiglu(x, w, n + ".mlp", spec["mlp"]["limit"])
            x = x + layer_norm(y, w[n + ".norm2"], w[n + ".norm2.b"], eps) * w[n + ".ls2"]
        if trace is not None:
            trace.append(x.clone())
    x = layer_norm(x, w["final.norm"], w["final.norm.b"], eps)
    cap = config["logit_softcap"]
    return cap * torch.tanh(x @ w["head"].T / cap)
