"""A plain, slow Sipelorn for tests: float64 NumPy, one function per mechanism.

It shares no code with `dynalm_b200`: it reads config.json and model.safetensors by itself. `PlainSipelorn.logits(tokens)`
runs a whole sequence at once, `logits(tokens, cuts=[...])` runs it in portions and `logits_stepwise(tokens)` token by
token, all from explicit state per layer: the keys and values (or latent records) seen so far, the last inputs of every
short convolution, the last token. They agree to rounding of float64.

Notation. W the stream's width. Attention: H query heads over G key/value heads, key size d, value size e, window w, taps
K of the convolutions, distance numbers (a, b) per head. Latent attention: H heads, d unrotated and r rotated numbers per
query, latent size R, value size e. Mixture: E experts in C groups of neighbours, `keep` groups and `top` experts a token.
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def xielu(z, p, q):
    """softplus(p) z^2 + z/2 above zero, (1/2 + softplus(q)) (e^z - 1 - z) + z/2 at and below it."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def layer_norm(x, weight, bias, eps):
    dev = x - x.mean(axis=-1, keepdims=True)
    return dev / np.sqrt((dev * dev).mean(axis=-1, keepdims=True) + eps) * weight + bias


def rms_norm(x, weight, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def bigram_rows(tokens, previous, table: dict):
    """Rows of the table of token pairs; `previous` None: the first token has nothing in front of it."""
    rows, last = [], previous
    for t in tokens:
        rows.append(table["buckets"] if last is None else (last * table["mul_prev"] + t * table["mul_cur"]) % table["buckets"])
        last = t
    return rows


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


def rotate_pairs(x, positions, freq, mag: float):
    """x [T, ..., n]; numbers 2i and 2i + 1 turn by position * freq[i], lengths times mag; the rest pass."""
    n = 2 * len(freq)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    shape = (len(ang),) + (1,) * (x.ndim - 2) + (len(freq),)
    c, s = (np.cos(ang) * mag).reshape(shape), (np.sin(ang) * mag).reshape(shape)
    y = x.copy()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2], y[..., 1:n:2] = u * c - v * s, v * c + u * s
    return y


def convolve(u, taps, kept):
    """u [T, channels] behind the kept inputs [K - 1, channels] (zeros at a start), taps [channels, K], the last one the
    current token's. Returns (result, the inputs to keep)."""
    K = taps.shape[1]
    full = np.concatenate([kept, u]) if K > 1 else u
    T = u.shape[0]
    y = sum(full[j:j + T] * taps[:, j] for j in range(K))
    return y, (full[len(full) - (K - 1):].copy() if K > 1 else kept)


def visible(i: int, j: int, window: int) -> bool:
    return 0 <= i - j and (window <= 0 or i - j < window)


def attend(q, k, v, q_pos, k_pos, scale, window=0, a=None, b=None):
    """q [Tq, H, d], k [Tk, G, d], v [Tk, G, e] -> [Tq, H, e]; a_h ln(1 + b_h * distance) comes off every score."""
    Tq, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((Tq, H, v.shape[2]))
    k_pos = np.asarray(k_pos)
    for t in range(Tq):
        js = np.array([x for x in range(len(k_pos)) if visible(q_pos[t], k_pos[x], window)])
        gap = q_pos[t] - k_pos[js]
        for h in range(H):
            g = h // (H // G)
            s = (k[js, g] @ q[t, h]) * scale
            if a is not None:
                s = s - a[h] * np.log(1.0 + b[h] * gap)
            w = np.exp(s - s.max())
            out[t, h] = (w[:, None] * v[js, g]).sum(0) / w.sum()
    return out


def route(z, correction, top: int, groups: int, keep: int):
    """Router logits z [E] -> (chosen experts, their weights): scores sigmoid(z), chosen by score + correction among the
    groups whose two largest choice scores sum highest, weighed by the score alone."""
    s = sigmoid(z)
    c = s + correction
    E = len(s)
    if groups > 1:
        per = E // groups
        best_two = np.sort(c.reshape(groups, per), axis=1)[:, -2:].sum(axis=1)
        kept = np.argsort(-best_two, kind="stable")[:keep]
        allowed = np.isin(np.arange(E) // per, kept)
        c = np.where(allowed, c, -np.inf)
    order = [int(i) for i in np.argsort(-c, kind="stable")[:top]]
    return order, s[order]


def gated_expert(x, gate, up, down):
    return down @ (silu(gate @ x) * (up @ x))


# --------------------------------------------------------------------------------------------
# the model
# --------------------------------------------------------------------------------------------

class PlainSipelorn:
    def __init__(self, folder: Optional[str] = None, config: Optional[dict] = None, tensors: Optional[dict] = None):
        if folder is not None:
            with open(os.path.join(folder, "config.json")) as f:
                config = json.load(f)
            tensors = read_tensors(os.path.join(folder, "model.safetensors"))
        self.cfg, self.t = config, {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
        self.eps = config["norm"]["eps"]

    # mixers over a run of tokens [T, W] at the given positions, from and into the layer's state
    def _attention(self, i, h, positions, states):
        m, t, p, st = self.cfg["layers"][i]["mixer"], self.t, f"l{i}.mix.", states[i]
        T = h.shape[0]
        H, G, d = m["heads"], m["kv_heads"], m["dim"]
        e = m["vdim"]

        def projected(name, heads, size):
            u = h @ t[p + name].T + t[p + name + ".b"]
            taps = t.get(p + name + ".conv")
            if taps is not None:
                kept = st.get("conv." + name, np.zeros((taps.shape[1] - 1, u.shape[1])))
                u, st["conv." + name] = convolve(u, taps, kept)
            return u.reshape(T, heads, size)
        q = projected("q", H, d)
        source = m.get("kv_from")
        if source is None:
            st.setdefault("k", []).extend(projected("k", G, d))
            st.setdefault("v", []).extend(projected("v", G, e))
            st.setdefault("pos", []).extend(positions)
            source = i
        kv = states[source]
        mask = m.get("mask")
        o = attend(q, np.array(kv["k"]), np.array(kv["v"]), positions, kv["pos"], m["scale"], mask["size"] if mask else 0,
                   t[p + "r1"], t[p + "r2"])
        o = o.reshape(T, H * e) * sigmoid(h @ t[p + "g"].T)
        return o @ t[p + "o"].T

    def _latent(self, i, h, positions, st):
        m, t, p = self.cfg["layers"][i]["mixer"], self.t, f"l{i}.mix."
        T = h.shape[0]
        H, d, r, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        freq, mag = yarn(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling")) if m.get("rot") else (np.zeros(0), 1.0)
        q = (h @ t[p + "q"].T).reshape(T, H, d + r)
        q = np.concatenate([q[..., :d], rotate_pairs(q[..., d:], positions, freq, mag)], axis=-1)
        low = h @ t[p + "dkv"].T
        st.setdefault("c", []).extend(rms_norm(low[:, :R], t[p + "dkv.norm"], self.eps))
        st.setdefault("kr", []).extend(rotate_pairs(low[:, R:], positions, freq, mag))
        st.setdefault("pos", []).extend(positions)
        c, kr = np.array(st["c"]), np.array(st["kr"])
        n = len(c)
        k = np.concatenate([(c @ t[p + "uk"].T).reshape(n, H, d), np.repeat(kr[:, None], H, axis=1)], axis=-1)
        v = (c @ t[p + "uv"].T).reshape(n, H, e)
        o = attend(q, k, v, positions, st["pos"], m["scale"])
        return o.reshape(T, H * e) @ t[p + "o"].T

    def _ffn(self, i, h):
        f, t, p = self.cfg["layers"][i]["mlp"], self.t, f"l{i}.mlp."
        if f["kind"] == "dense":
            a = t[p + "act"]
            return xielu(h @ t[p + "up"].T, a[0], a[1]) @ t[p + "down"].T
        r = f["router"]
        groups = r.get("groups") or {}
        out = np.zeros_like(h)
        for n in range(h.shape[0]):
            chosen, w = route(t[p + "router"] @ h[n], t[p + "correction"], r["top"], groups.get("count", 1), groups.get("keep", 1))
            for j, wj in zip(chosen, w):
                out[n] += wj * gated_expert(h[n], t[f"{p}e{j}.gate"], t[f"{p}e{j}.up"], t[f"{p}e{j}.down"])
            if f.get("shared"):
                out[n] += sigmoid(t[p + "shared.sg"] @ h[n]) * gated_expert(h[n], t[p + "shared.gate"], t[p + "shared.up"], t[p + "shared.down"])
        return out

    def run(self, tokens, positions, states, last: dict, layers_out: Optional[list] = None):
        """A run of tokens through every layer from and into `states` (one dict per layer) and `last` (the last token);
        returns the stream [T, W]."""
        t, cfg = self.t, self.cfg
        tokens = [int(x) for x in tokens]
        emb = cfg.get("embedding") or {}
        x = t["embed"][tokens] * emb.get("scale", 1.0)
        pairs = emb.get("bigram")
        if pairs:
            x = x + t["bigram"][bigram_rows(tokens, last.get("token"), pairs)]
        last["token"] = tokens[-1]
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            h = layer_norm(x, t[p + "norm1"], t[p + "norm1.b"], self.eps)
            y = self._attention(i, h, list(positions), states) if layer["type"] == "attention" else \
                self._latent(i, h, list(positions), states[i])
            x = x + sigmoid(h @ t[p + "rg1"].T + t[p + "rg1.b"]) * y
            if layer.get("mlp") is not None:
                h = layer_norm(x, t[p + "norm2"], t[p + "norm2.b"], self.eps)
                x = x + sigmoid(h @ t[p + "rg2"].T + t[p + "rg2.b"]) * self._ffn(i, h)
            side = cfg.get("token_side")
            if side:
                n = side["dim"]
                e = t["side.embed"][tokens][:, i * n:(i + 1) * n]
                y = (gelu_tanh(x @ t[p + "side.gate"].T) * e) @ t[p + "side.proj"].T
                x = x + rms_norm(y, t[p + "side.norm"], self.eps)
            if layers_out is not None:
                layers_out.append(x.copy())
        return x

    def head(self, x):
        return layer_norm(x, self.t["final.norm"], self.t["final.norm.b"], self.eps) @ self.t["head"].T

    def logits(self, tokens, layers: bool = False, cuts: Optional[List[int]] = None):
        """Logits [T, vocab] of a sequence fed whole, or in portions of the sizes `cuts` (the rest in one piece)."""
        states, last = [dict() for _ in self.cfg["layers"]], {}
        at, rows, per_layer = 0, [], []
        for size in list(cuts or []) + [len(tokens)]:
            size = min(size, len(tokens) - at)
            if size <= 0:
                continue
            part = [] if layers else None
            rows.append(self.head(self.run(tokens[at:at + size], range(at, at + size), states, last, part)))
            if layers:
                per_layer.append(part)
            at += size
        out = np.concatenate(rows)
        if layers:
            return out, [np.concatenate([part[i] for part in per_layer]) for i in range(len(self.cfg["layers"]))]
        return out

    def logits_stepwise(self, tokens):
        return self.logits(tokens, cuts=[1] * len(tokens))
