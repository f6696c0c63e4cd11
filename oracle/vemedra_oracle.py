"""Plain, slow restatement of the Vemedra decoder: one function per mechanism, whole sequences, no cache.

Every function takes and returns CPU tensors of one floating type (float64 in the tests) and works on one
sequence ``[tokens, ...]`` that starts at position 0.  Recurrences are written as loops over tokens and
attention as loops over query positions, straight from the definitions, so that nothing here shares structure
(let alone code) with the CUDA path.  The tests compare the framework with it."""
from __future__ import annotations

import math

import torch


def rms_norm(x, eps, weight=None):
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def causal_conv(h, taps_weight):
    """Depthwise: out[t, c] = sum_j w[c, j] h[t - taps + 1 + j, c], nothing before the start."""
    T, C = h.shape
    taps = taps_weight.shape[1]
    out = torch.zeros_like(h)
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] += taps_weight[:, j] * h[src]
    return out


def rotate(x, base, dims):
    """x [T, heads, dim]: the first ``dims`` dimensions turn in pairs (i, i + dims/2) by position * base^(-2i/dims)."""
    T = x.shape[0]
    y = x.clone()
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        for p in range(T):
            c, s = math.cos(p * f), math.sin(p * f)
            u, v = x[p, :, i], x[p, :, i + dims // 2]
            y[p, :, i] = u * c - v * s
            y[p, :, i + dims // 2] = v * c + u * s
    return y


def chunk_attention(q, k, v, scale, softcap, chunk, sink):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim].  A query sees the keys at or before it in its
    own chunk of ``chunk`` positions; tanh-capped scores; exp(sink[h]) joins the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        lo = (t // chunk) * chunk
        for h in range(H):
            g = h // (H // G)
            s = (k[lo:t + 1, g] @ q[t, h]) * scale
            s = softcap * torch.tanh(s / softcap)
            m = torch.maximum(s.max(), sink[h])
            e = torch.exp(s - m)
            out[t, h] = (e / (e.sum() + torch.exp(sink[h] - m))) @ v[lo:t + 1, g]
    return out


def retention(q, k, v, decay):
    """q, k [T, heads, dim], v [T, heads, vdim], decay [heads] -> o [T, heads, vdim] (k already scaled)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    d = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def min_gru(z_logit, u):
    """z_logit, u [T, width] (biases included) -> the states S [T, width]."""
    z = torch.sigmoid(z_logit)
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S = torch.zeros_like(u[0])
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = (1 - z[t]) * S + z[t] * cand[t]
        out[t] = S
    return out


def silu(x):
    return x * torch.sigmoid(x)


def clamped_glu(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


class VemedraOracle:
    def __init__(self, config: dict, tensors: dict, dtype=torch.float64):
        self.c = config
        self.w = {k: v.to(dtype) for k, v in tensors.items()}
        self.dtype = dtype

    def mixer_mingru(self, p, m, h):
        w = self.w
        S = min_gru(h @ w[p + "z"].T + w[p + "z.b"], h @ w[p + "x"].T + w[p + "x.b"])
        return (S * silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def mixer_attention(self, p, m, h):
        w, T = self.w, h.shape[0]
        q = rotate((h @ w[p + "q"].T).view(T, m["heads"], m["dim"]), m["rot"]["base"], m["rot"]["dims"])
        k = rotate((h @ w[p + "k"].T).view(T, m["kv_heads"], m["dim"]), m["rot"]["base"], m["rot"]["dims"])
        v = (h @ w[p + "v"].T).view(T, m["kv_heads"], m["vdim"])
        o = chunk_attention(q, k, v, m["scale"], m["softcap"], m["mask"]["size"], w[p + "sink"])
        return o.reshape(T, -1) @ w[p + "o"].T

    def mixer_retention(self, p, m, h):
        w, T = self.w, h.shape[0]
        q = (h @ w[p + "q"].T).view(T, m["heads"], m["dim"])
        k = (h @ w[p + "k"].T).view(T, m["heads"], m["dim"]) * m["dim"] ** -0.5
        v = (h @ w[p + "v"].T).view(T, m["heads"], m["vdim"])
        o = rms_norm(retention(q, k, v, m["decay"]), self.c["norm"]["eps"])
        return (o.reshape(T, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def mixer(self, p, layer, h):
        m = layer["mixer"]
        if layer["type"] == "mingru":
            return self.mixer_mingru(p, m, h)
        assert layer["type"] == "parallel"
        return (m["left_scale"] * self.mixer_attention(p + "left.", m["left"], h)
                + m["right_scale"] * self.mixer_retention(p + "right.", m["right"], h))

    def sublayer_input(self, x, norm, conv):
        h = rms_norm(x, self.c["norm"]["eps"], self.w[norm])
        return h + causal_conv(h, self.w[conv])

    def layer(self, i, x):
        lay, p, w = self.c["layers"][i], f"l{i}.", self.w
        x = x + self.mixer(p + "mix.", lay, self.sublayer_input(x, p + "norm1", p + "canon1"))
        if lay["mlp"] is not None:
            h = self.sublayer_input(x, p + "norm2", p + "canon2")
            y = clamped_glu(h @ w[p + "mlp.gate"].T, h @ w[p + "mlp.up"].T, lay["mlp"]["limit"])
            x = x + y @ w[p + "mlp.down"].T
        return x

    def forward(self, tokens, layers_out=None):
        """Logits of every position of one sequence, [T, vocab]."""
        loop = self.c.get("loop")
        x0 = x = self.w["embed"][torch.as_tensor(tokens)]
        n = len(self.c["layers"])
        start, stop, times = (loop["start"], loop["stop"], loop["times"]) if loop else (0, 0, 0)

        def run(i, x):
            x = self.layer(i, x)
            if layers_out is not None:
                layers_out.append(x)
            return x
        for i in range(start):
            x = run(i, x)
        for t in range(times):
            if t > 0:
                x = x + x0
            x = x + self.w["loop.step"][t]
            for i in range(start, stop):
                x = run(i, x)
        for i in range(stop, n):
            x = run(i, x)
        return rms_norm(x, self.c["norm"]["eps"], self.w["final.norm"]) @ self.w["head"].T
