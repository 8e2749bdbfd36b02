"""Configurations of models described layer by layer, with different sequence mixers and an optional
loop over some of the layers (the Ralapel design), for `Decoder`.

No counterpart in the reference, whose decoders are attention-only.  `LayeredConfig.from_json`
reads a checkpoint's config.json; every size and constant comes from it.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

MIXERS = {"latent_attention": 1, "delta": 2, "mamba2": 3}   # cg_mixer (include/catgrad_cuda.h)


class LayerStruct(C.Structure):
    """Mirror of `cg_layer_config` (include/catgrad_cuda.h)."""
    _fields_ = [("mixer", C.c_int32), ("ffn", C.c_int32), ("act", C.c_int32), ("heads", C.c_int32), ("kv_heads", C.c_int32),
                ("dim", C.c_int32), ("rot_dim", C.c_int32), ("vdim", C.c_int32), ("kv_rank", C.c_int32), ("state", C.c_int32),
                ("groups", C.c_int32), ("norm_groups", C.c_int32), ("conv", C.c_int32), ("rot_base", C.c_double), ("scale", C.c_double)]


class LoopStruct(C.Structure):
    """Mirror of `cg_loop_config`."""
    _fields_ = [("start", C.c_int32), ("stop", C.c_int32), ("times", C.c_int32)]


@dataclass
class LayerSpec:
    """One layer: the mixer's name, its sizes (the keys config.json uses) and the feed-forward width
    (0 = the layer has none)."""
    mixer: str
    sizes: dict
    ffn: int = 0
    act: int = 1   # 0 silu, 1 tanh gelu

    def struct(self) -> LayerStruct:
        s, m = LayerStruct(), self.sizes
        s.mixer, s.ffn, s.act = MIXERS[self.mixer], self.ffn, self.act
        s.heads, s.vdim = m["heads"], m["vdim"]
        if self.mixer == "latent_attention":
            s.dim, s.rot_dim, s.kv_rank, s.scale = m["dim"], m["rot_dim"], m["kv_rank"], m["scale"]
            s.rot_base = m["rot"]["base"] if m["rot_dim"] else 0.0
        elif self.mixer == "delta":
            s.dim, s.kv_heads, s.conv = m["dim"], m["kv_heads"], m["conv"]
        else:
            s.state, s.groups, s.norm_groups, s.conv = m["state"], m["groups"], m["norm_groups"], m["conv"]
        return s


@dataclass
class LayeredConfig:
    name: str
    hidden_size: int
    vocab_size: int
    layers: list[LayerSpec]
    loop: tuple[int, int, int] | None = None   # (start, stop, times)
    rms_norm_eps: float = 1e-6
    dtype: str = "bf16"
    arch: str = "layered"
    extras: dict = field(default_factory=dict)

    @classmethod
    def from_json(cls, d: dict) -> "LayeredConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            mlp = e.get("mlp")
            if mlp and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            if e["type"] == "latent_attention" and e["mixer"]["rot_dim"] and e["mixer"]["rot"]["dims"] != e["mixer"]["rot_dim"]:
                raise ValueError(f"layer {i}: the rotated part must be rotated whole")
            layers.append(LayerSpec(e["type"], e["mixer"], mlp["ff"] if mlp else 0))
        lp = d.get("loop")
        return cls(d.get("architecture", "layered"), d["width"], d["vocab"], layers,
                   (lp["start"], lp["stop"], lp["times"]) if lp else None, d["norm"]["eps"])

    def layer_runs(self) -> list[int]:
        """Layers in the order they run."""
        n = len(self.layers)
        if not self.loop:
            return list(range(n))
        a, b, t = self.loop
        return list(range(a)) + list(range(a, b)) * t + list(range(b, n))

    def param_shapes(self) -> dict[str, tuple[int, ...]]:
        """Tensor names and shapes of a checkpoint (weights [out, in])."""
        W = self.hidden_size
        s = {"embed": (self.vocab_size, W), "embed.norm": (W,), "final.norm": (W,), "head": (self.vocab_size, W)}
        if self.loop:
            s["loop.in"] = (W, 2 * W)
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L.sizes
            H, dv = m["heads"], m["vdim"]
            s[p + "norm1"] = s[p + "norm1b"] = (W,)
            if L.ffn:
                s[p + "norm2"] = s[p + "norm2b"] = (W,)
                s[p + "mlp.gate"] = s[p + "mlp.up"] = (L.ffn, W)
                s[p + "mlp.down"] = (W, L.ffn)
            p += "mix."
            s[p + "o"] = (W, H * dv)
            if L.mixer == "latent_attention":
                d, r, R = m["dim"], m["rot_dim"], m["kv_rank"]
                s[p + "q"], s[p + "dkv"], s[p + "dkv.norm"] = (H * (d + r), W), (R + r, W), (R,)
                s[p + "uk"], s[p + "uv"] = (H * d, R), (H * dv, R)
            elif L.mixer == "delta":
                K, d, taps = m["kv_heads"], m["dim"], m["conv"]
                for n, rows in (("q", K * d), ("k", K * d), ("v", H * dv)):
                    s[p + n], s[p + n + ".conv"] = (rows, W), (rows, taps)
                s[p + "b"] = s[p + "a"] = (H, W)
                s[p + "g"] = (H * dv, W)
                s[p + "A_log"] = s[p + "dt_bias"] = (H,)
                s[p + "norm"] = (dv,)
            else:
                N, G, taps = m["state"], m["groups"], m["conv"]
                ch = H * dv + 2 * G * N
                s[p + "in"], s[p + "conv"], s[p + "conv.b"] = (H * dv + ch + H, W), (ch, taps), (ch,)
                s[p + "A_log"] = s[p + "dt_bias"] = s[p + "D"] = (H,)
                s[p + "norm"] = (H * dv,)
        return s

    @staticmethod
    def synthetic(name: str) -> tuple[float, float]:
        """(mean, std) a synthetic checkpoint draws a tensor with: gains 1, slow decays, wide taps."""
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "A_log":
            return 0.5, 0.5
        if leaf == "dt_bias":
            return -3.0, 1.0
        if name.endswith("conv"):
            return 0.0, 0.4
        if name.endswith("conv.b"):
            return 0.0, 0.1
        if leaf in ("D", "norm", "norm1", "norm1b", "norm2", "norm2b"):
            return 1.0, 0.0
        return 0.0, 0.02


def bench_shape(name: str, width: int, ff: int, vocab: int) -> LayeredConfig:
    """A Ralapel-shaped model at a real model's widths, for measurements: per mixer the head sizes
    larger models use (128 x 128 delta states, 128 x 64 Mamba-2 states with one group, latent rows
    of 512 + 32), a loop over three of the layers."""
    ssd = LayerSpec("mamba2", {"heads": 2 * width // 64, "groups": 1, "state": 128, "vdim": 64, "norm_groups": 1, "conv": 4})
    lat = LayerSpec("latent_attention", {"heads": width // 128, "dim": 96, "rot_dim": 32, "vdim": 128, "kv_rank": 512, "scale": 128 ** -0.5,
                                         "rot": {"base": 10000.0, "dims": 32}}, ff)
    dlt = LayerSpec("delta", {"heads": width // 64, "kv_heads": width // 128, "dim": 128, "vdim": 128, "conv": 4}, ff)
    return LayeredConfig(name, width, vocab, [ssd, lat, dlt, ssd, lat, dlt, ssd, dlt], (1, 4, 2))


RALAPEL_W1024 = bench_shape("ralapel-w1024-shape", 1024, 4096, 32000)
RALAPEL_W2048 = bench_shape("ralapel-w2048-shape", 2048, 8192, 128256)
RALAPEL_W4096 = bench_shape("ralapel-w4096-shape", 4096, 14336, 128256)
