"""Plain double-precision Gitozen model over checkpoint tensors by name, one function per mechanism, one sequence at a
time and without any cache: every function sees the whole sequence.  Shares no code with the package."""
import math

import torch
import torch.nn.functional as F


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def causal_conv(x, w):
    """x [n, channels], w [channels, taps], last tap on the current row; silu."""
    n, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + padded[j:j + n] * w[:, j]
    return F.silu(y)


def delta_recurrence(q, k, v, g, beta, state=None):
    """q, k, g [n, heads, dim], v [n, heads, vdim], beta [n, heads] -> outputs [n, heads, vdim], final state."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(n):
        for h in range(H):
            Sh = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - Sh.T @ k[t, h])
            S[h] = Sh + torch.outer(k[t, h], u)
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def decay(pre, a_log, dt_bias, heads):
    """Per head and key channel: exp(-exp(A_log) softplus(pre + dt_bias)); pre [n, heads * dim]."""
    sp = F.softplus(pre + dt_bias).view(pre.shape[0], heads, -1)
    return torch.exp(-torch.exp(a_log)[None, :, None] * sp)


def delta_mixer(h, T, p, m, eps):
    n, H, KV = h.shape[0], m.heads, m.kv_heads
    q = causal_conv(h @ T(p + "q").T, T(p + "q.conv")).view(n, KV, m.dim)
    k = causal_conv(h @ T(p + "k").T, T(p + "k.conv")).view(n, KV, m.dim)
    v = causal_conv(h @ T(p + "v").T, T(p + "v.conv")).view(n, H, m.vdim)
    share = [i // (H // KV) for i in range(H)]
    q, k = (unit(q) / math.sqrt(m.dim))[:, share], unit(k)[:, share]
    beta = torch.sigmoid(h @ T(p + "b").T)
    g = decay((h @ T(p + "a1").T) @ T(p + "a2").T, T(p + "A_log"), T(p + "dt_bias"), H)
    o, _ = delta_recurrence(q, k, v, g, beta)
    gate = torch.sigmoid((h @ T(p + "g1").T) @ T(p + "g2").T).view(n, H, m.vdim)
    return (rms(o, eps) * T(p + "norm") * gate).reshape(n, -1) @ T(p + "o").T


def causal_attention(q, k, v, scale):
    """q, k [n, heads, dim], v [n, heads, vdim]."""
    n = q.shape[0]
    out = torch.zeros(n, q.shape[1], v.shape[2], dtype=q.dtype)
    for i in range(n):
        s = torch.einsum("hd,jhd->hj", q[i], k[:i + 1]) * scale
        out[i] = torch.einsum("hj,jhv->hv", torch.softmax(s, -1), v[:i + 1])
    return out


def latent_mixer(h, T, p, m, eps):
    n, H = h.shape[0], m.heads
    q = (h @ T(p + "q").T).view(n, H, m.dim)
    c = rms(h @ T(p + "dkv").T, eps) * T(p + "dkv.norm")
    k, v = (c @ T(p + "uk").T).view(n, H, m.dim), (c @ T(p + "uv").T).view(n, H, m.vdim)
    o = causal_attention(q, k, v, m.scale) * torch.sigmoid(h @ T(p + "g").T)[:, :, None]
    return o.reshape(n, -1) @ T(p + "o").T


def choose_experts(scores, s):
    """Indices of the `top` best experts inside the `keep` groups with the best single expert, per row."""
    size = s.experts // s.groups
    rows = []
    for r in scores.tolist():
        best = sorted(range(s.groups), key=lambda g: (-max(r[g * size:(g + 1) * size]), g))[:s.keep]
        allowed = [e for g in best for e in range(g * size, (g + 1) * size)]
        rows.append(sorted(allowed, key=lambda e: (-r[e], e))[:s.top])
    return rows


def experts(h, T, p, s):
    scores = torch.softmax(h @ T(p + "router").T, -1)
    out = torch.zeros_like(h)
    for t, chosen in enumerate(choose_experts(scores, s)):
        for e in chosen:
            q = f"{p}e{e}."
            z = F.silu(h[t] @ T(q + "gate").T) * (h[t] @ T(q + "up").T)
            out[t] += scores[t, e] * (z @ T(q + "down").T)
    return out


class Oracle:
    def __init__(self, cfg, tensors):
        self.cfg, self.cache, self.tensors = cfg, {}, tensors

    def T(self, name):
        if name not in self.cache:
            self.cache[name] = self.tensors(name).double().cpu()
        return self.cache[name]

    def layers(self, tokens):
        """Residual stream after every layer."""
        cfg, T = self.cfg, self.T
        x = T("embed")[torch.tensor(tokens)]
        out = []
        for i, l in enumerate(cfg.layers):
            p = f"l{i}."
            h = rms(x, cfg.norm_eps) * T(p + "norm1")
            mixer = delta_mixer if hasattr(l.mixer, "taps") else latent_mixer
            y = mixer(h, T, p + "mix.", l.mixer, cfg.norm_eps) * torch.sigmoid(h @ T(p + "rg1").T + T(p + "rg1.b"))
            if l.mlp is not None:
                y = y + experts(h, T, p + "mlp.", l.mlp) * torch.sigmoid(h @ T(p + "rg2").T + T(p + "rg2.b"))
            x = x + y
            out.append(x)
        return out

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self.cache:
            z = (rms(self.layers(tokens)[-1], self.cfg.norm_eps) * self.T("final.norm")) @ self.T("head").T
            cap = self.cfg.logit_softcap
            self.cache[key] = cap * torch.tanh(z / cap) if cap else z
        return self.cache[key]

    def greedy(self, prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(self.logits(seq)[-1].argmax()))
        return seq[len(prompt):]
