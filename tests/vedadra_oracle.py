"""Plain double-precision Vedadra model over checkpoint tensors by name, one function per mechanism, one sequence at a time
and without any cache: every function sees the whole sequence.  Shares no code with the package."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_rms(x, w, groups, eps):
    """Every one of `groups` equal consecutive parts of a row divided by its own root mean square."""
    n = x.shape[-1] // groups
    out = torch.empty_like(x)
    for g in range(groups):
        out[..., g * n:(g + 1) * n] = rms(x[..., g * n:(g + 1) * n], eps)
    return out * w


def window(n, size, keep_first=0):
    """[n, n] visibility: the key at j for the query at i."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def slope(h, heads):
    return 2.0 ** (-8.0 * (h + 1) / heads)


def raw_scores(q, k, scale):
    """q [n, H, dim], k [n, G, dim] -> [H, n, n]; a query head meets the key head of its group."""
    H, G = q.shape[1], k.shape[1]
    return torch.stack([q[:, h] @ k[:, h // (H // G)].T * scale for h in range(H)])


def distance_bias(heads, n):
    i, j = torch.arange(n)[:, None], torch.arange(n)[None]
    return torch.stack([slope(h, heads) * (i - j).double() for h in range(heads)])


def mix_scores(s, T):
    """score_h <- sum_g T[h, g] score_g."""
    out = torch.zeros_like(s)
    for h in range(s.shape[0]):
        for g in range(s.shape[0]):
            out[h] += T[h, g] * s[g]
    return out


def attend(s, v, visible):
    """s [H, n, n], v [n, G, vdim] -> [n, H, vdim]."""
    H, G = s.shape[0], v.shape[1]
    w = torch.softmax(s.masked_fill(~visible, -math.inf), -1)
    return torch.stack([w[h] @ v[:, h // (H // G)] for h in range(H)], 1)


def talking_mixer(h, T, p, m, eps):
    n, H, G = h.shape[0], m.heads, m.kv_heads
    q = (h @ T(p + "q").T + T(p + "q.b")).view(n, H, m.dim)
    k = (h @ T(p + "k").T + T(p + "k.b")).view(n, G, m.dim)
    v = k
    q, k = rms(q, eps) * T(p + "q.norm"), rms(k, eps) * T(p + "k.norm")
    s = raw_scores(q, k, m.scale) * T(p + "temp")[:, None, None] - distance_bias(H, n)
    o = attend(mix_scores(s, T(p + "talk")), v, window(n, m.window, m.keep_first)).reshape(n, -1)
    return (o * torch.sigmoid(h @ T(p + "g").T)) @ T(p + "o").T + T(p + "o.b")


def map_weight(T, p, diff):
    dot = lambda a, b: torch.exp((T(p + a) * T(p + b)).sum())
    return dot("lq1", "lk1") - dot("lq2", "lk2") + diff


def map_difference(a1, a2, weight, diff, eps):
    return rms(a1 - weight * a2, eps) * (1 - diff)


def differential_mixer(h, T, p, m, eps):
    n, H, G = h.shape[0], m.heads, m.kv_heads
    q = rms((h @ T(p + "q").T).view(n, H, 2, m.dim), eps) * T(p + "q.norm")
    k = rms((h @ T(p + "k").T).view(n, G, 2, m.dim), eps) * T(p + "k.norm")
    v = (h @ T(p + "v").T).view(n, G, m.vdim)
    vis = window(n, m.window, m.keep_first)
    a1, a2 = (attend(raw_scores(q[:, :, i], k[:, :, i], m.scale), v, vis) for i in (0, 1))
    return map_difference(a1, a2, map_weight(T, p, m.diff), m.diff, eps).reshape(n, -1) @ T(p + "o").T


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_ff(x, T, p):
    return (gelu_tanh(x @ T(p + "gate").T) * (x @ T(p + "up").T)) @ T(p + "down").T


def run_order(n_layers, loop):
    """(layer, whether a later pass begins here) in the order a token passes them."""
    if loop is None:
        return [(i, False) for i in range(n_layers)]
    out = [(i, False) for i in range(loop.start)]
    for t in range(loop.times):
        out += [(i, t > 0 and i == loop.start) for i in range(loop.start, loop.stop)]
    return out + [(i, False) for i in range(loop.stop, n_layers)]


class Oracle:
    def __init__(self, cfg, tensors):
        self.cfg, self.cache, self.tensors = cfg, {}, tensors

    def T(self, name):
        if name not in self.cache:
            self.cache[name] = self.tensors(name).double().cpu()
        return self.cache[name]

    def norm(self, x, name):
        return group_rms(x, self.T(name), self.cfg.norm_groups, self.cfg.norm_eps)

    def layers(self, tokens):
        """Residual stream after every layer run."""
        cfg, T, eps = self.cfg, self.T, self.cfg.norm_eps
        x = embedded = T("embed")[torch.tensor(tokens)]
        out = []
        for i, again in run_order(len(cfg.layers), cfg.loop):
            l, p = cfg.layers[i], f"l{i}."
            if again:
                x = x + embedded
            mixer = talking_mixer if l.mixer.kind == "attention" else differential_mixer
            x = x + self.norm(mixer(self.norm(x, p + "norm1"), T, p + "mix.", l.mixer, eps), p + "norm1b")
            if l.mlp is not None:
                x = x + self.norm(gated_ff(self.norm(x, p + "norm2"), T, p + "mlp."), p + "norm2b")
            out.append(x)
        return out

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self.cache:
            self.cache[key] = self.norm(self.layers(tokens)[-1], "final.norm") @ self.T("head").T
        return self.cache[key]

    def greedy(self, prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(self.logits(seq)[-1].argmax()))
        return seq[len(prompt):]
