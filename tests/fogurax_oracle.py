"""Plain, slow restatement of the Fogurax design for the tests: one function per mechanism, straight from the equations, in
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


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def linear(x, w, name):
    y = x @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


def causal_conv(u, taps):
    """Every channel: the value d tokens back weighs with the d-th tap from the end; nothing lies before the first token."""
    y = torch.zeros_like(u)
    for d, tap in enumerate(taps.flip(1).T):
        if d < len(u):
            y[d:] += tap * u[:len(u) - d]
    return y


# ---- rotations
def plain_frequencies(rot):
    return [rot["base"] ** (-2 * i / rot["dims"]) for i in range(rot["dims"] // 2)]


def band_frequencies(rot):
    """Long waves slower by ``factor``, short ones kept, a blend between."""
    s, out = rot["scaling"], []
    for f in plain_frequencies(rot):
        wave = 2 * math.pi / f
        if wave < s["original"] / s["high"]:
            out.append(f)
        elif wave > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            mix = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1 - mix) * f / s["factor"] + mix * f)
    return out


def yarn_frequencies(rot):
    s, dims, out = rot["scaling"], rot["dims"], []

    def channel(turns):
        return dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(rot["base"]))

    lo, hi = max(math.floor(channel(s["fast"])), 0), min(math.ceil(channel(s["slow"])), dims - 1)
    for i, f in enumerate(plain_frequencies(rot)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1 - ramp))
    return out


def yarn_amplitude(rot):
    return 0.1 * math.log(rot["scaling"]["factor"]) + 1


def rotate(x, frequencies, amplitude, interleaved):
    """x [t, h, d]: pairs (2i, 2i+1) or (i, i + n) of the first 2n channels, turned by position times frequency."""
    n = len(frequencies)
    a = torch.arange(len(x), dtype=torch.float64)[:, None] * torch.tensor(frequencies, dtype=torch.float64)
    c, s = (amplitude * f(a).to(x.dtype)[:, None] for f in (torch.cos, torch.sin))
    first, second = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if interleaved else (slice(0, n), slice(n, 2 * n))
    out = x.clone()
    out[..., first] = x[..., first] * c - x[..., second] * s
    out[..., second] = x[..., second] * c + x[..., first] * s
    return out


# ---- which keys are seen
def seen_causal(t):
    i, j = torch.arange(t)[:, None], torch.arange(t)[None]
    return j <= i


def seen_window(t, size):
    i, j = torch.arange(t)[:, None], torch.arange(t)[None]
    return (j <= i) & (i - j < size)


def seen_chunk(t, size):
    i, j = torch.arange(t)[:, None], torch.arange(t)[None]
    return (j <= i) & (i // size == j // size)


def attend(q, k, v, scale, seen):
    """Grouped softmax attention: q [t, H, d], k [t, G, d], v [t, G, e] -> [t, H, e]."""
    n = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(n, 1), v.repeat_interleave(n, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    return torch.einsum("hij,jhe->ihe", torch.softmax(s.masked_fill(~seen, -math.inf), -1), v)


def heads(x, n):
    return x.view(len(x), n, -1)


def head_gate(o, h, w, name):
    return o * torch.sigmoid(linear(h, w, name + ".g"))[..., None]


# ---- mixers
def conv_attention(h, w, name, mix, eps):
    """'attention': biases, short convolutions, interleaved rotation with banded frequencies, unit norm after it, head gate."""
    q, k, v = (causal_conv(linear(h, w, f"{name}.{n}"), w[f"{name}.{n}.conv"]) for n in "qkv")
    f = band_frequencies(mix["rot"])
    q = rms(rotate(heads(q, mix["heads"]), f, 1.0, True), eps)
    k = rms(rotate(heads(k, mix["kv_heads"]), f, 1.0, True), eps)
    o = attend(q, k, heads(v, mix["kv_heads"]), mix["scale"], seen_causal(len(h)))
    return linear(head_gate(o, h, w, name).flatten(1), w, name + ".o")


def normed_qkv(h, w, name, mix, eps):
    """Projections, q and k divided by the root mean square over all heads."""
    q = rms(linear(h, w, name + ".q"), eps) * w[name + ".q.norm"]
    k = rms(linear(h, w, name + ".k"), eps) * w[name + ".k.norm"]
    return heads(q, mix["heads"]), heads(k, mix["kv_heads"]), heads(linear(h, w, name + ".v"), mix["kv_heads"])


def chunk_attention(h, w, name, mix, eps):
    """'attention_2': norm over the projection, half-split rotation with YaRN, chunks."""
    q, k, v = normed_qkv(h, w, name, mix, eps)
    f, a = yarn_frequencies(mix["rot"]), yarn_amplitude(mix["rot"])
    o = attend(rotate(q, f, a, False), rotate(k, f, a, False), v, mix["scale"], seen_chunk(len(h), mix["mask"]["size"]))
    return linear(o.flatten(1), w, name + ".o")


def window_attention(h, w, name, mix, eps):
    """Left half of 'parallel': norm over the projection, interleaved rotation, sliding window, head gate."""
    q, k, v = normed_qkv(h, w, name, mix, eps)
    f = plain_frequencies(mix["rot"])
    o = attend(rotate(q, f, 1.0, True), rotate(k, f, 1.0, True), v, mix["scale"], seen_window(len(h), mix["mask"]["size"]))
    return linear(head_gate(o, h, w, name).flatten(1), w, name + ".o")


def previous(h):
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def channel_decay(m, w, name):
    """Per token and key channel, in (0, 1)."""
    return torch.exp(-torch.exp(linear(torch.tanh(linear(m, w, name + ".w1")), w, name + ".w2") + w[name + ".w0"]))


def time_mix_scan(r, k, v, decay, u):
    """A matrix per head, read before the token is written into it, the token itself through the bonus;  r, k, decay [t, h, d], v [t, h, e]."""
    S, out = k.new_zeros(k.shape[1], k.shape[2], v.shape[2]), []
    for i in range(len(r)):
        kv = k[i][:, :, None] * v[i][:, None, :]
        out.append(torch.einsum("hde,hd->he", S + u[:, :, None] * kv, r[i]))
        S = decay[i][:, :, None] * S + kv
    return torch.stack(out)


def time_mix(h, w, name, mix, eps):
    """Right half of 'parallel': RWKV-style recurrence with a decay per key channel and a bonus for the current token."""
    back, H = previous(h), mix["heads"]
    m = {s: h + (back - h) * w[f"{name}.mu.{s}"] for s in "rkvgw"}
    r, k, v = (heads(linear(m[s], w, f"{name}.{s}"), H) for s in "rkv")
    o = time_mix_scan(r, k, v, heads(channel_decay(m["w"], w, name), H), w[name + ".u"])
    return linear(rms(o, eps).flatten(1) * w[name + ".norm"] * silu(linear(m["g"], w, name + ".g")), w, name + ".o")


def side_by_side(h, w, name, mix, eps):
    left = window_attention(h, w, name + ".left", mix["left"], eps)
    return mix["left_scale"] * left + mix["right_scale"] * time_mix(h, w, name + ".right", mix["right"], eps)


MIXERS = {"attention": conv_attention, "attention_2": chunk_attention, "parallel": side_by_side}


# ---- feed-forwards
def gated_unit(h, w, name):
    return linear(silu(linear(h, w, name + ".gate")) * linear(h, w, name + ".up"), w, name + ".down")


def route(z, top):
    """Chosen experts and their sigmoid scores [t, top]."""
    s = torch.sigmoid(z)
    best = torch.sort(s, dim=-1, descending=True, stable=True).indices[:, :top]
    return best, torch.gather(s, -1, best)


def experts(h, w, name, mlp):
    """Scores multiply the experts' inputs; one expert sees every token as it is."""
    best, p = route(linear(h, w, name + ".router"), mlp["router"]["top"])
    out = gated_unit(h, w, name + ".shared")
    for e in range(mlp["router"]["experts"]):
        t, j = (best == e).nonzero(as_tuple=True)
        out[t] += gated_unit(p[t, j, None] * h[t], w, f"{name}.e{e}")
    return out


def feed_forward(h, w, name, mlp):
    return gated_unit(h, w, name) if mlp["kind"] == "dense" else experts(h, w, name, mlp)


def token_side(x, e, w, name, eps):
    """The layer's own part ``e`` of the token's side embedding, gated by the stream."""
    y = linear(gelu_tanh(linear(x, w, name + ".gate")) * e, w, name + ".proj")
    return rms(y, eps) * w[name + ".norm"]


def forward(tokens, w, config, trace=None):
    """Logits [t, vocab] of one sequence; ``trace`` (a list) receives the residual stream after every layer."""
    eps, m, tokens = config["norm"]["eps"], config["residual_mult"], torch.as_tensor(tokens)
    n = config["token_side"]["dim"]
    x, side = w["embed"][tokens], w["side.embed"][tokens]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        h = rms(x, eps) * w[p + ".norm1"]
        y = MIXERS[layer["type"]](h, w, p + ".mix", layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + feed_forward(h, w, p + ".mlp", layer["mlp"])
        x = x + m * y
        x = x + m * token_side(x, side[:, i * n:(i + 1) * n], w, p + ".side", eps)
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T
