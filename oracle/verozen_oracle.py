"""Plain, slow restatement of the Verozen decoder: one function per mechanism, whole sequences, no cache.

Every function takes and returns CPU tensors of one floating type (float64 in the tests) and works on one sequence
``[tokens, ...]`` that starts at position 0.  Recurrences are loops over tokens, attention is a loop over query
positions and the experts are visited token by token, straight from the definitions, so that nothing here shares
structure (let alone code) with the CUDA path.  The tests compare the framework with it."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """x over its root mean square (last dimension)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def group_norm(x, groups, eps, weight):
    """Each of ``groups`` consecutive parts of the vector over its own root mean square, then the weight."""
    parts = [rms(part, eps) for part in x.chunk(groups, dim=-1)]
    return torch.cat(parts, dim=-1) * weight


def silu(x):
    return x * torch.sigmoid(x)


def gelu_erf(x):
    return 0.5 * x * (1 + torch.erf(x / math.sqrt(2.0)))


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def rotate(x, base, dims, interleaved):
    """x [T, heads, dim]: the first ``dims`` dimensions turn in pairs by position * base^(-2i/dims); pair i is (2i, 2i + 1)
    where ``interleaved``, else (i, i + dims/2)."""
    y = x.clone()
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        f = base ** (-2.0 * i / dims)
        for p in range(x.shape[0]):
            c, s = math.cos(p * f), math.sin(p * f)
            u, v = x[p, :, a], x[p, :, b]
            y[p, :, a] = u * c - v * s
            y[p, :, b] = v * c + u * s
    return y


def sigmoid_attention(q, k, v, scale, temp, bias):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim].  Key j <= t has the weight
    sigmoid(scale temp[h] q.k + bias[h]); the weights are not normalised."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            out[t, h] = torch.sigmoid((k[:t + 1, g] @ q[t, h]) * scale * temp[h] + bias[h]) @ v[:t + 1, g]
    return out


def decayed_linear_attention(q, k, v, decay):
    """q, k [T, heads, dim], v [T, heads, vdim], decay [T, heads, dim] (per key channel) -> o [T, heads, vdim]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def route(z, correction, top, group_count, group_keep, scale):
    """Router logits z [experts] of one token -> {expert: weight}."""
    s = torch.sigmoid(z)
    choice = s + correction
    size = len(z) // group_count
    score = []
    for g in range(group_count):
        best = sorted(choice[g * size:(g + 1) * size].tolist(), reverse=True)
        score.append(sum(best[:2]))
    kept = sorted(range(group_count), key=lambda g: -score[g])[:group_keep]
    allowed = [e for e in range(len(z)) if e // size in kept]
    chosen = sorted(allowed, key=lambda e: -float(choice[e]))[:top]
    total = sum(s[e] for e in chosen) + 1e-20
    return {e: s[e] / total * scale for e in chosen}


def experts(h, weights, ups, downs):
    """h [T, width]; ``weights[t]`` as ``route`` gives them; up [ff, width] and down [width, ff] of every expert."""
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in weights[t].items():
            out[t] += w * (downs[e] @ gelu_erf(ups[e] @ h[t]))
    return out


def side_input(x, e, gate, proj, norm, eps):
    """What a layer's token input e [T, dim] adds to x [T, width]."""
    return rms((gelu_tanh(x @ gate.T) * e) @ proj.T, eps) * norm


class VerozenOracle:
    def __init__(self, config: dict, tensors: dict, dtype=torch.float64):
        self.c = config
        self.w = {k: v.to(dtype) for k, v in tensors.items()}
        self.eps = config["norm"]["eps"]

    def norm(self, x, name):
        return group_norm(x, self.c["norm"]["groups"], self.eps, self.w[name])

    def mixer_gla(self, p, m, h):
        w, T, H, D = self.w, h.shape[0], m["heads"], m["dim"]
        q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
        k = (h @ w[p + "k"].T).view(T, H, D)
        v = (h @ w[p + "v"].T).view(T, H, m["vdim"])
        z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
        o = decayed_linear_attention(q, k, v, (torch.sigmoid(z) ** (1.0 / m["tau"])).view(T, H, D))
        o = rms(o, self.eps) * w[p + "norm"]
        return (o.reshape(T, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def mixer_attention(self, p, m, h):
        w, T = self.w, h.shape[0]
        q = (h @ w[p + "q"].T).view(T, m["heads"], m["dim"])
        k = (h @ w[p + "k"].T).view(T, m["kv_heads"], m["dim"])
        rot = m["rot"]
        qr = rotate(rms(q, self.eps) * w[p + "q.norm"], rot["base"], rot["dims"], True)
        kr = rotate(rms(k, self.eps) * w[p + "k.norm"], rot["base"], rot["dims"], True)
        o = sigmoid_attention(qr, kr, k, m["scale"], w[p + "temp"], w[p + "pb"])
        return o.reshape(T, -1) @ w[p + "o"].T

    def mixer_retention(self, p, m, h):
        w, T, H, D, rot = self.w, h.shape[0], m["heads"], m["dim"], m["rot"]
        q = rotate((h @ w[p + "q"].T).view(T, H, D), rot["base"], rot["dims"], False)
        k = rotate((h @ w[p + "k"].T).view(T, H, D), rot["base"], rot["dims"], False) * D ** -0.5
        v = (h @ w[p + "v"].T).view(T, H, m["vdim"])
        decay = torch.tensor(m["decay"], dtype=h.dtype)[None, :, None].expand(T, H, D)
        o = rms(decayed_linear_attention(q, k, v, decay), self.eps)
        return (o.reshape(T, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def feed_forward(self, p, f, h):
        r, w = f["router"], self.w
        z = h @ w[p + "router"].T
        picks = [route(z[t], w[p + "correction"], r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"]) for t in range(len(h))]
        return experts(h, picks, [w[f"{p}e{e}.up"] for e in range(r["experts"])], [w[f"{p}e{e}.down"] for e in range(r["experts"])])

    def layer(self, i, x, tokens):
        lay, p, w, alpha = self.c["layers"][i], f"l{i}.", self.w, self.c["postln_alpha"]
        mixer = {"gla": self.mixer_gla, "attention": self.mixer_attention, "retention": self.mixer_retention}[lay["type"]]
        x = self.norm(alpha * x + mixer(p + "mix.", lay["mixer"], x), p + "norm1")
        if lay["mlp"] is not None:
            x = self.norm(alpha * x + self.feed_forward(p + "mlp.", lay["mlp"], x), p + "norm2")
        n = self.c["token_side"]["dim"]
        e = w["side.embed"][tokens][:, i * n:(i + 1) * n]
        return x + side_input(x, e, w[p + "side.gate"], w[p + "side.proj"], w[p + "side.norm"], self.eps)

    def forward(self, tokens, layers_out=None):
        """Logits of every position of one sequence, [T, vocab]."""
        tokens = torch.as_tensor(tokens)
        x = self.w["embed"][tokens]
        for i in range(len(self.c["layers"])):
            x = self.layer(i, x, tokens)
            if layers_out is not None:
                layers_out.append(x)
        return self.norm(x, "final.norm") @ self.w["head"].T
