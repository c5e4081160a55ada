"""A plain, slow Nisotar for tests: float64 NumPy, one function per mechanism.

It shares no code with `dynalm_b200`: it reads config.json and model.safetensors by itself. `PlainNisotar.logits(tokens)`
runs a whole sequence at once, `logits(tokens, cuts=[...])` runs it in portions and `logits_stepwise(tokens)` token by
token, all from explicit state per layer: the keys and values (or latent records) seen so far, the matrix states of the
delta rule, the last inputs of every short convolution. They agree to rounding of float64.

Notation. W the stream's width. Attention: H query heads over G key/value heads, key size d, value size e, window w or
chunk c. Latent attention: H heads, d unrotated and r rotated numbers per query, latent size R, value size e. Delta rule: H
heads with states d x e over G query/key heads, K taps, inner sizes of the decay's and the gate's projections read from
their tensors. Mixture: E experts, `top` a token.
"""

from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import numpy as np


def read_tensors(path: str) -> Dict[str, np.ndarray]:
    """A safetensors file: 8-byte little-endian header length, JSON header, data. Floats come back as float64."""
    with open(path, "rb") as f:
        raw = f.read()
    (hlen,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + hlen])
    data = raw[8 + hlen:]
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        lo, hi = e["data_offsets"]
        buf = data[lo:hi]
        if e["dtype"] == "F32":
            a = np.frombuffer(buf, dtype="<f4").astype(np.float64)
        elif e["dtype"] == "BF16":
            a = (np.frombuffer(buf, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif e["dtype"] == "I32":
            a = np.frombuffer(buf, dtype="<i4").copy()
        else:
            raise ValueError(f"dtype {e['dtype']} of {name}")
        out[name] = a.reshape(e["shape"])
    return out


# --------------------------------------------------------------------------------------------
# mechanisms
# --------------------------------------------------------------------------------------------

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, dtype=np.float64)))


def softplus(z):
    return np.logaddexp(0.0, z)


def silu(z):
    return z * sigmoid(z)


def layer_norm(x, weight, eps):
    dev = x - x.mean(axis=-1, keepdims=True)
    return dev / np.sqrt((dev * dev).mean(axis=-1, keepdims=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def yarn(base: float, dims: int, scaling: Optional[dict]):
    """(one frequency per pair, the factor on cos and sin). With `scaling` {factor, original, fast, slow} the frequencies
    that turn fewer than `slow` times over `original` positions are divided by factor, those that turn more than `fast`
    times stay, and a linear ramp over the pairs lies in between."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    s, L = scaling["factor"], scaling["original"]

    def pair_of(turns):
        return dims * math.log(L / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s * ramp + f * (1.0 - ramp), 0.1 * math.log(s) + 1.0


def rotate_halves(x, positions, freq, mag: float = 1.0):
    """x [T, ..., n]; numbers i and i + len(freq) turn by position * freq[i], lengths times mag; those from 2 len(freq) on
    pass."""
    n = len(freq)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    shape = (len(ang),) + (1,) * (x.ndim - 2) + (n,)
    c, s = (np.cos(ang) * mag).reshape(shape), (np.sin(ang) * mag).reshape(shape)
    y = x.copy()
    u, v = x[..., :n], x[..., n:2 * n]
    y[..., :n], y[..., n:2 * n] = u * c - v * s, v * c + u * s
    return y


def convolve(u, taps, kept):
    """u [T, channels] behind the kept inputs [K - 1, channels] (zeros at a start), taps [channels, K], the last one the
    current token's. Returns (result, the inputs to keep)."""
    K = taps.shape[1]
    full = np.concatenate([kept, u]) if K > 1 else u
    T = u.shape[0]
    y = sum(full[j:j + T] * taps[:, j] for j in range(K))
    return y, (full[len(full) - (K - 1):].copy() if K > 1 else kept)


def visible(i: int, j: int, window: int = 0, chunk: int = 0) -> bool:
    """Whether position i sees key j: no later one, inside the window where there is one, of the same chunk where
    sequences are cut into chunks."""
    if j > i:
        return False
    if window > 0 and i - j >= window:
        return False
    return chunk <= 0 or i // chunk == j // chunk


def attend(q, k, v, q_pos, k_pos, scale, window=0, chunk=0, sink=False):
    """q [Tq, H, d], k [Tk, G, d], v [Tk, G, e] -> [Tq, H, e]; with `sink` one more exp(0) in the denominator."""
    Tq, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((Tq, H, v.shape[2]))
    for t in range(Tq):
        js = np.array([x for x in range(len(k_pos)) if visible(q_pos[t], k_pos[x], window, chunk)])
        for h in range(H):
            g = h // (H // G)
            s = (k[js, g] @ q[t, h]) * scale
            top = max(s.max(), 0.0) if sink else s.max()
            w = np.exp(s - top)
            out[t, h] = (w[:, None] * v[js, g]).sum(0) / (w.sum() + (np.exp(-top) if sink else 0.0))
    return out


def delta_step(S, q, k, v, g, beta):
    """One token of one head: S [d, e], q, k, g [d], v [e] -> (S, o). The rows of S are scaled by g, then corrected along k,
    then read along q."""
    S = g[:, None] * S
    u = beta * (v - S.T @ k)
    S = S + np.outer(k, u)
    return S, S.T @ q


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def half_sum(a, b, wa, wb, eps):
    return 0.5 * (rms_norm(a, wa, eps) + rms_norm(b, wb, eps))


def clamped_gate(g, u, limit):
    """min(g, limit) sigmoid(1.702 min(g, limit)) (clamp(u) + 1)."""
    g = np.minimum(g, limit)
    return g * sigmoid(1.702 * g) * (np.clip(u, -limit, limit) + 1.0)


def route(z, top: int):
    """Router logits z [E] -> (the `top` largest, softmax over those alone)."""
    order = [int(i) for i in np.argsort(-z, kind="stable")[:top]]
    w = np.exp(z[order] - z[order].max())
    return order, w / w.sum()


def gated_expert(x, gate, up, down):
    return down @ (silu(gate @ x) * (up @ x))


# --------------------------------------------------------------------------------------------
# the model
# --------------------------------------------------------------------------------------------

class PlainNisotar:
    def __init__(self, folder: Optional[str] = None, config: Optional[dict] = None, tensors: Optional[dict] = None):
        if folder is not None:
            with open(os.path.join(folder, "config.json")) as f:
                config = json.load(f)
            tensors = read_tensors(os.path.join(folder, "model.safetensors"))
        self.cfg, self.t = config, {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
        self.eps = config["norm"]["eps"]

    # mixers over a run of tokens [T, W] at the given positions, from and into a state
    def _attention(self, m, p, h, positions, st, chunked: bool):
        t, T = self.t, h.shape[0]
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        q = (h @ t[p + "q"].T).reshape(T, H, d)
        k = (h @ t[p + "k"].T).reshape(T, G, d)
        v = k if chunked else (h @ t[p + "v"].T).reshape(T, G, e)
        q, k = rms_norm(q, t[p + "q.norm"], self.eps), rms_norm(k, t[p + "k.norm"], self.eps)
        rot = m.get("rot")
        if rot:
            freq, mag = yarn(rot["base"], rot["dims"], rot.get("scaling"))
            q, k = rotate_halves(q, positions, freq, mag), rotate_halves(k, positions, freq, mag)
        st.setdefault("k", []).extend(k)
        st.setdefault("v", []).extend(v)
        st.setdefault("pos", []).extend(positions)
        size = m["mask"]["size"] if m.get("mask") else 0
        o = attend(q, np.array(st["k"]), np.array(st["v"]), positions, st["pos"], m["scale"], window=0 if chunked else size,
                   chunk=size if chunked else 0, sink=True)
        return o.reshape(T, -1) @ t[p + "o"].T

    def _delta(self, m, p, h, st):
        t, T = self.t, h.shape[0]
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

        def projected(name, heads, size):
            u, taps = h @ t[p + name].T, t[p + name + ".conv"]
            kept = st.get("conv." + name, np.zeros((taps.shape[1] - 1, u.shape[1])))
            u, st["conv." + name] = convolve(u, taps, kept)
            return silu(u).reshape(T, heads, size)
        q, k, v = projected("q", G, d), projected("k", G, d), projected("v", H, e)
        q, k = unit(q) * d ** -0.5, unit(k)
        beta = sigmoid(h @ t[p + "b"].T)
        rate = np.exp(t[p + "A_log"])[None, :, None]
        g = np.exp(-rate * softplus((h @ t[p + "a1"].T) @ t[p + "a2"].T + t[p + "dt_bias"]).reshape(T, H, d))
        gate = sigmoid((h @ t[p + "g1"].T) @ t[p + "g2"].T).reshape(T, H, e)
        S = st.setdefault("S", np.zeros((H, d, e)))
        o = np.zeros((T, H, e))
        for n in range(T):
            for i in range(H):
                j = i // (H // G)
                S[i], o[n, i] = delta_step(S[i], q[n, j], k[n, j], v[n, i], g[n, i], beta[n, i])
        return (rms_norm(o, t[p + "norm"], self.eps) * gate).reshape(T, H * e) @ t[p + "o"].T

    def _parallel(self, m, p, h, positions, st):
        a = self._attention(m["left"], p + "left.", h, positions, st.setdefault("left", {}), chunked=True)
        b = self._delta(m["right"], p + "right.", h, st.setdefault("right", {}))
        return half_sum(a, b, self.t[p + "left.out"], self.t[p + "right.out"], self.eps)

    def _latent(self, m, p, h, positions, st):
        t, T = self.t, h.shape[0]
        H, d, r, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        rot = m.get("rot")
        freq, mag = yarn(rot["base"], rot["dims"], rot.get("scaling")) if rot else (np.zeros(0), 1.0)
        q = (h @ t[p + "q"].T).reshape(T, H, d + r)
        q = np.concatenate([q[..., :d], rotate_halves(q[..., d:], positions, freq, mag)], axis=-1)
        low = h @ t[p + "dkv"].T
        st.setdefault("c", []).extend(rms_norm(low[:, :R], t[p + "dkv.norm"], self.eps))
        st.setdefault("kr", []).extend(rotate_halves(low[:, R:], positions, freq, mag))
        st.setdefault("pos", []).extend(positions)
        c, kr = np.array(st["c"]), np.array(st["kr"])
        n = len(c)
        k = np.concatenate([(c @ t[p + "uk"].T).reshape(n, H, d), np.repeat(kr[:, None], H, axis=1)], axis=-1)
        v = (c @ t[p + "uv"].T).reshape(n, H, e)
        o = attend(q, k, v, positions, st["pos"], m["scale"], window=m["mask"]["size"] if m.get("mask") else 0)
        return o.reshape(T, H * e) @ t[p + "o"].T

    def _ffn(self, f, p, h):
        t = self.t
        if f["kind"] == "dense":
            a = clamped_gate(h @ t[p + "gate"].T + t[p + "gate.b"], h @ t[p + "up"].T + t[p + "up.b"], f["limit"])
            return a @ t[p + "down"].T + t[p + "down.b"]
        out = np.zeros_like(h)
        for n in range(h.shape[0]):
            chosen, w = route(t[p + "router"] @ h[n] + t[p + "router.b"], f["router"]["top"])
            for j, wj in zip(chosen, w):
                out[n] += wj * gated_expert(h[n], t[f"{p}e{j}.gate"], t[f"{p}e{j}.up"], t[f"{p}e{j}.down"])
        return out

    def run(self, tokens, positions, states, layers_out: Optional[list] = None):
        """A run of tokens through every layer from and into `states` (one dict per layer); returns the stream [T, W]."""
        t, cfg = self.t, self.cfg
        positions = list(positions)
        x = t["embed"][[int(n) for n in tokens]] * (cfg.get("embedding") or {}).get("scale", 1.0)
        for i, layer in enumerate(cfg["layers"]):
            p, m, st = f"l{i}.mix.", layer["mixer"], states[i]
            h = layer_norm(x, t[f"l{i}.norm1"], self.eps)
            if layer["type"] == "parallel":
                x = x + self._parallel(m, p, h, positions, st)
            elif layer["type"] == "attention":
                x = x + self._attention(m, p, h, positions, st, chunked=False)
            else:
                x = x + self._latent(m, p, h, positions, st)
            if layer.get("mlp") is not None:
                x = x + self._ffn(layer["mlp"], f"l{i}.mlp.", layer_norm(x, t[f"l{i}.norm2"], self.eps))
            if layers_out is not None:
                layers_out.append(x.copy())
        return x

    def head(self, x):
        return layer_norm(x, self.t["final.norm"], self.eps) @ self.t["head"].T

    def logits(self, tokens, layers: bool = False, cuts: Optional[List[int]] = None):
        """Logits [T, vocab] of a sequence fed whole, or in portions of the sizes `cuts` (the rest in one piece)."""
        states = [dict() for _ in self.cfg["layers"]]
        at, rows, per_layer = 0, [], []
        for size in list(cuts or []) + [len(tokens)]:
            size = min(size, len(tokens) - at)
            if size <= 0:
                continue
            part = [] if layers else None
            rows.append(self.head(self.run(tokens[at:at + size], range(at, at + size), states, part)))
            if layers:
                per_layer.append(part)
            at += size
        out = np.concatenate(rows)
        if layers:
            return out, [np.concatenate([part[i] for part in per_layer]) for i in range(len(self.cfg["layers"]))]
        return out

    def logits_stepwise(self, tokens):
        return self.logits(tokens, cuts=[1] * len(tokens))
