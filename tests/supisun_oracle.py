"""Plain double-precision Supisun model over checkpoint tensors by name, one function per mechanism, one sequence at a
time and without any cache: every function sees the whole sequence.  Shares no code with the package."""
import math

import torch
import torch.nn.functional as F


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def causal_conv(x, w, bias=None):
    """x [n, channels], w [channels, taps]: the last tap meets the current row, zeros come before the first."""
    n, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x) if bias is None else bias.expand_as(x).clone()
    for t in range(n):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] += w[:, j] * x[t - taps + 1 + j]
    return y


def rotate(x, base, dims):
    """x [n, heads, dim]; row t is at position t; coordinates i and i + dims / 2 of the first `dims` turn together."""
    out, half = x.clone(), dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = t * base ** (-2.0 * i / dims)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * math.cos(a) - v * math.sin(a)
            out[t, :, i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def chunk_attention(q, k, v, scale, size):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim]: softmax over the keys up to the query's own in its own chunk."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n):
        lo = i // size * size
        for h in range(H):
            g = h // (H // G)
            w = torch.softmax(k[lo:i + 1, g] @ q[i, h] * scale, 0)
            out[i, h] = w @ v[lo:i + 1, g]
    return out


def attention_mixer(h, T, p, m, eps, first_values):
    """`first_values`: a dict the first value-mixing layer leaves its values in."""
    n = h.shape[0]
    q = (rms(h @ T(p + "q").T, eps) * T(p + "q.norm")).view(n, m.heads, m.dim)
    k = (rms(h @ T(p + "k").T, eps) * T(p + "k.norm")).view(n, m.kv_heads, m.dim)
    v = rms((h @ T(p + "v").T).view(n, m.kv_heads, m.vdim), eps)
    q, k = rotate(q, m.rot_base, m.rot_dims), rotate(k, m.rot_base, m.rot_dims)
    if m.v_mix:
        if "v" in first_values:
            lam = T(p + "vmix")
            v = (1 - lam) * v + lam * first_values["v"]
        else:
            first_values["v"] = v
    return chunk_attention(q, k, v, m.scale, m.chunk).reshape(n, -1) @ T(p + "o").T


def selective_scan(x, dt, A, B, C, D, state=None):
    """x, dt [n, inner], A [inner, N], B, C [n, N], D [inner] -> outputs [n, inner], final state [inner, N]."""
    S = torch.zeros_like(A) if state is None else state.clone()
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out, S


def mamba_mixer(h, T, p, m):
    xz = h @ T(p + "in").T
    x, z = xz[:, :m.inner], xz[:, m.inner:]
    x = F.silu(causal_conv(x, T(p + "conv"), T(p + "conv.b")))
    low = x @ T(p + "x").T
    dt, B, C = low[:, :m.dt_rank], low[:, m.dt_rank:m.dt_rank + m.state], low[:, m.dt_rank + m.state:]
    dt = F.softplus(dt @ T(p + "dt").T + T(p + "dt.b"), threshold=1e9)
    y, _ = selective_scan(x, dt, -torch.exp(T(p + "A_log")), B, C, T(p + "D"))
    return (y * F.silu(z)) @ T(p + "o").T


def delta_recurrence(q, k, v, g, beta, state=None):
    """q, k [n, heads, dim], v [n, heads, vdim], g, beta [n, heads] -> outputs [n, heads, vdim], final state."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(n):
        for h in range(H):
            Sh = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - Sh.T @ k[t, h])
            S[h] = Sh + torch.outer(k[t, h], u)
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def head_decay(pre, a_log, dt_bias):
    return torch.exp(-torch.exp(a_log) * F.softplus(pre + dt_bias, threshold=1e9))


def delta_mixer(h, T, p, m, eps):
    n, H, KV = h.shape[0], m.heads, m.kv_heads
    part = lambda name: F.silu(causal_conv(h @ T(p + name).T, T(p + name + ".conv")))
    share = [i // (H // KV) for i in range(H)]
    q = (unit(part("q").view(n, KV, m.dim)) / math.sqrt(m.dim))[:, share]
    k = unit(part("k").view(n, KV, m.dim))[:, share]
    v = part("v").view(n, H, m.vdim)
    beta = torch.sigmoid(h @ T(p + "b").T)
    g = head_decay(h @ T(p + "a").T, T(p + "A_log"), T(p + "dt_bias"))
    o, _ = delta_recurrence(q, k, v, g, beta)
    gate = F.silu(h @ T(p + "g").T).view(n, H, m.vdim)
    return (rms(o, eps) * T(p + "norm") * gate).reshape(n, -1) @ T(p + "o").T


def dense_ff(x, T, p):
    z = x @ T(p + "up").T
    return (0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))) @ T(p + "down").T


class Oracle:
    def __init__(self, cfg, tensors):
        self.cfg, self.cache, self.tensors = cfg, {}, tensors

    def T(self, name):
        if name not in self.cache:
            self.cache[name] = self.tensors(name).double().cpu()
        return self.cache[name]

    def layers(self, tokens):
        """Residual stream after every layer."""
        cfg, T, eps = self.cfg, self.T, self.cfg.norm_eps
        x = T("embed")[torch.tensor(tokens)] + T("pos")[:len(tokens)]
        out, values = [], {}
        for i, l in enumerate(cfg.layers):
            p = f"l{i}."
            h = x + causal_conv(x, T(p + "canon1"))
            if l.mixer.kind == "attention":
                y = attention_mixer(h, T, p + "mix.", l.mixer, eps, values)
            elif l.mixer.kind == "mamba1":
                y = mamba_mixer(h, T, p + "mix.", l.mixer)
            else:
                y = delta_mixer(h, T, p + "mix.", l.mixer, eps)
            x = x + layer_norm(y, T(p + "norm1"), T(p + "norm1.b"), eps)
            if l.mlp is not None:
                x = x + layer_norm(dense_ff(x, T, p + "mlp."), T(p + "norm2"), T(p + "norm2.b"), eps)
            out.append(x)
        return out

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self.cache:
            x = self.layers(tokens)[-1]
            self.cache[key] = layer_norm(x, self.T("final.norm"), self.T("final.norm.b"), self.cfg.norm_eps) @ self.T("head").T
        return self.cache[key]

    def greedy(self, prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(self.logits(seq)[-1].argmax()))
        return seq[len(prompt):]
