"""Configurations of models described layer by layer: different sequence mixers and feed-forwards, an
optional loop over some of the layers, and what a design fixes for all of them (the Ralapel, Segedra,
Regupel and Kivorax designs), for `Decoder`.

No counterpart in the reference, whose decoders are attention-only.  `LayeredConfig.from_json`
reads a checkpoint's config.json; every size and constant comes from it.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

MIXERS = {"latent_attention": 1, "delta": 2, "mamba2": 3, "attention": 4, "lightning": 5,   # cg_mixer (include/catgrad_cuda.h)
          "channel_delta": 6, "gla": 7, "rglru": 8}
SILU, GELU, BOUNDED, RELU2, GELU1 = range(5)                                                      # cg_act
RECURRENT = ("delta", "mamba2", "lightning", "channel_delta", "gla", "rglru")


class LayerStruct(C.Structure):
    """Mirror of `cg_layer_config` (include/catgrad_cuda.h)."""
    _fields_ = [("mixer", C.c_int32), ("ffn", C.c_int32), ("act", C.c_int32), ("heads", C.c_int32), ("kv_heads", C.c_int32),
                ("dim", C.c_int32), ("rot_dim", C.c_int32), ("vdim", C.c_int32), ("kv_rank", C.c_int32), ("state", C.c_int32),
                ("groups", C.c_int32), ("norm_groups", C.c_int32), ("conv", C.c_int32), ("window", C.c_int32), ("qk_norm", C.c_int32),
                ("sink", C.c_int32), ("experts", C.c_int32), ("top_k", C.c_int32), ("correction", C.c_int32), ("scoring", C.c_int32),
                ("weigh_input", C.c_int32), ("shared_ffn", C.c_int32), ("keep_first", C.c_int32), ("rot_half", C.c_int32), ("gate", C.c_int32),
                ("weights_of", C.c_int32), ("dist_bias", C.c_int32), ("out_norm", C.c_int32), ("rot_base", C.c_double), ("rot_factor", C.c_double), ("rot_low", C.c_double),
                ("rot_high", C.c_double), ("rot_original", C.c_double), ("scale", C.c_double), ("router_scale", C.c_double),
                ("act_limit", C.c_double), ("out_scale", C.c_double), ("q_temp_coef", C.c_double), ("q_temp_every", C.c_double),
                ("tau", C.c_double), ("decay", C.c_void_p), ("beside", C.c_void_p)]


class LoopStruct(C.Structure):
    """Mirror of `cg_loop_config`."""
    _fields_ = [("start", C.c_int32), ("stop", C.c_int32), ("times", C.c_int32)]


@dataclass(frozen=True)
class AttentionTraits:
    """What a design's attention has besides its sizes."""
    qk_norm: int = 0             # 1: norms over all query and over all key heads; 2: per head, without gains
    sink: bool = False           # a learned term of the softmax's denominator per head
    gate: bool = False           # a head's output times the sigmoid of a projection, one number per head
    wide_gate: bool = False      # the same with a number per value
    dist_bias: bool = False      # a logarithm of the distance is taken off the scores, with two learned numbers per head
    rot_half: bool = False       # component i is rotated with component i + dims / 2, not with its neighbour


@dataclass(frozen=True)
class Routing:
    """How a design's experts are chosen, weighted and built."""
    act: int
    correction: bool = False     # a learned number per expert is added for the choice
    sigmoid: bool = False        # scores are the sigmoids of the logits, not their softmax
    weigh_input: bool = False    # the weights multiply the experts' inputs

    @property
    def gated(self) -> bool:
        """Whether an expert has a gate projection."""
        return self.act != RELU2


@dataclass(frozen=True)
class Design:
    """What a family of layer-by-layer models fixes for all its layers."""
    mixers: tuple[str, ...]
    dense_act: int | None        # of dense feed-forwards; None: there are none
    routing: Routing | None = None   # feed-forwards may be mixtures of experts
    pre_norms: bool = True       # norms before the sublayers
    post_norms: bool = False     # norms behind the sublayers
    layer_norm: bool = False     # layer and final norms take the mean off and add a bias
    embed_norm: bool = False
    loop_input: bool = False     # a loop's passes start from W [x; normed embedding]
    norm_plus_one: bool = False  # layer and final norms multiply by 1 + w
    tied_head: bool = False
    attention: AttentionTraits = AttentionTraits()
    beside: tuple[str, str] | None = None   # mixers of the "parallel" type, left and right
    beside_norms: bool = False   # each of their results has a norm, and the mean of both counts
    parallel_sublayers: bool = False   # one norm per layer, read by mixer and feed-forward, which are added together
    depth_average: bool = False  # behind every layer a learned weighted sum over all results so far
    left: AttentionTraits = AttentionTraits()   # of the attention among them

    def switches(self) -> dict[str, int]:
        """Fields of `cg_decoder_config`."""
        return {"post_norms": 0 if not self.post_norms else 1 if self.pre_norms else 2, "layer_norm": int(self.layer_norm),
                "embed_norm": int(self.embed_norm), "loop_input": int(self.loop_input), "norm_plus_one": int(self.norm_plus_one),
                "tie_embeddings": int(self.tied_head), "parallel_sublayers": int(self.parallel_sublayers),
                "depth_average": int(self.depth_average)}

    def norms(self, q: int) -> list[str]:
        """Names of the norms around sublayer q of a layer."""
        names = [f"norm{q}"] + ([f"norm{q}b"] if self.pre_norms and self.post_norms else [])
        return [n + b for n in names for b in (("", ".b") if self.layer_norm else ("",))]


DESIGNS = {
    "Ralapel": Design(("latent_attention", "delta", "mamba2"), GELU, post_norms=True, embed_norm=True, loop_input=True),
    "Segedra": Design(("attention",), RELU2, Routing(BOUNDED, correction=True), norm_plus_one=True, tied_head=True,
                      attention=AttentionTraits(qk_norm=1, sink=True)),
    "Regupel": Design(("attention", "parallel"), None, Routing(SILU, sigmoid=True, weigh_input=True), pre_norms=False, post_norms=True,
                      layer_norm=True, tied_head=True, attention=AttentionTraits(qk_norm=2, sink=True, gate=True, rot_half=True),
                      beside=("attention", "lightning"), left=AttentionTraits(qk_norm=1)),
    "Kivorax": Design(("parallel", "channel_delta", "gla"), GELU1, Routing(RELU2), beside=("attention", "rglru"),
                      left=AttentionTraits(wide_gate=True, dist_bias=True), beside_norms=True, parallel_sublayers=True, depth_average=True),
}


@dataclass
class Experts:
    """A mixture-of-experts feed-forward: `top` of `count` experts per token, their scores times `scale` the
    weights; `limit` bounds their units where the design has that; `shared` is the width of one more
    expert that every token runs (0: none)."""
    count: int
    top: int
    scale: float = 1.0
    limit: float = 0.0
    shared: int = 0


@dataclass
class LayerSpec:
    """One layer: the mixer's name, its sizes (the keys config.json uses) and the feed-forward width
    (of one expert if there are experts; 0 = the layer has none).  With `weights_of` the layer has no
    parameters of its own but those of that layer."""
    mixer: str
    sizes: dict
    ffn: int = 0
    act: int = GELU
    experts: Experts | None = None
    weights_of: int | None = None

    @property
    def window(self) -> int:
        """Tokens an attention layer sees, itself included; 0 = all before it."""
        return (self.sizes.get("mask") or {}).get("size") or 0

    @property
    def kept(self) -> int:
        """First tokens that stay visible beyond the window."""
        return (self.sizes.get("mask") or {}).get("keep_first") or 0

    @property
    def rotated(self) -> int:
        """Rotated components of an attention head."""
        return (self.sizes.get("rot") or {}).get("dims", 0)

    def parts(self, design: Design) -> list[tuple[str, "LayerSpec", AttentionTraits]]:
        """(prefix of the tensors, single mixer, traits if it is attention)."""
        if self.mixer != "parallel":
            return [("", self, design.attention)]
        return [(f"{side}.", LayerSpec(kind, self.sizes[side]), design.left) for side, kind in zip(("left", "right"), design.beside)]

    def struct(self, design: Design) -> LayerStruct:
        """The returned struct points into ones it keeps alive (`keep`)."""
        if self.mixer == "parallel":
            s, right = (p.mixer_struct(t) for _, p, t in self.parts(design))
            if design.beside_norms:
                s.out_norm = 1
            else:
                s.out_scale, right.out_scale = self.sizes["left_scale"], self.sizes["right_scale"]
            s.beside = C.addressof(right)
            s.keep = [right]
        else:
            s = self.mixer_struct(design.attention)
        s.ffn, s.act = self.ffn, self.act
        s.weights_of = 0 if self.weights_of is None else self.weights_of + 1
        if self.experts:
            e, r = self.experts, design.routing
            s.experts, s.top_k, s.router_scale, s.act_limit, s.shared_ffn = e.count, e.top, e.scale, e.limit, e.shared
            s.correction, s.scoring, s.weigh_input = int(r.correction), int(r.sigmoid), int(r.weigh_input)
        return s

    def mixer_struct(self, traits: AttentionTraits) -> LayerStruct:
        s, m = LayerStruct(), self.sizes
        s.mixer = MIXERS[self.mixer]
        if self.mixer == "rglru":
            if m["width"] % m["blocks"]:
                raise ValueError("equal blocks of channels")
            s.heads, s.vdim, s.conv = m["blocks"], m["width"] // m["blocks"], m["conv"]
            return s
        s.heads, s.vdim = m["heads"], m["vdim"]
        if self.mixer == "attention":
            s.dim, s.kv_heads, s.scale, s.window, s.keep_first = m["dim"], m["kv_heads"], m["scale"], self.window, self.kept
            s.rot_dim, s.rot_base = self.rotated, m["rot"]["base"] if self.rotated else 0.0
            scaling = (m.get("rot") or {}).get("scaling")
            if scaling:
                s.rot_factor, s.rot_low, s.rot_high, s.rot_original = (scaling[k] for k in ("factor", "low", "high", "original"))
            s.qk_norm, s.sink, s.rot_half, s.dist_bias = traits.qk_norm, int(traits.sink), int(traits.rot_half), int(traits.dist_bias)
            s.gate = 2 if traits.wide_gate else int(traits.gate)
            temp = m.get("q_temp")
            if temp:
                s.q_temp_coef, s.q_temp_every = temp["coef"], temp["every"]
        elif self.mixer == "lightning":
            if len(m["decay"]) != m["heads"]:
                raise ValueError("a decay per head")
            s.dim = m["dim"]
            s.keep = (C.c_double * m["heads"])(*m["decay"])
            s.decay = C.addressof(s.keep)
        elif self.mixer == "latent_attention":
            s.dim, s.rot_dim, s.kv_rank, s.scale = m["dim"], m["rot_dim"], m["kv_rank"], m["scale"]
            s.rot_base = m["rot"]["base"] if m["rot_dim"] else 0.0
        elif self.mixer in ("delta", "channel_delta"):
            s.dim, s.kv_heads, s.conv = m["dim"], m["kv_heads"], m["conv"]
        elif self.mixer == "gla":
            s.dim, s.tau = m["dim"], m["tau"]
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
    design: Design = DESIGNS["Ralapel"]
    streams: int = 0                           # rows of the residual stream per token; 0 = a plain one
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    token_side: int = 0                        # values per layer of the tokens' second embedding
    ranks: tuple[int, int] = (16, 16)          # of low-rank decays and gates, where no checkpoint's tensors give them
    extras: dict = field(default_factory=dict)

    @classmethod
    def from_json(cls, d: dict) -> "LayeredConfig":
        name = d["architecture"]
        design = DESIGNS[name]
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in design.mixers:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            mlp, of = e.get("mlp"), e.get("weights_of")
            if mlp and not ((mlp["kind"] == "dense" and design.dense_act is not None) or (mlp["kind"] == "moe" and design.routing)):
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            if e["type"] == "latent_attention" and e["mixer"]["rot_dim"] and e["mixer"]["rot"]["dims"] != e["mixer"]["rot_dim"]:
                raise ValueError(f"layer {i}: the rotated part must be rotated whole")
            seen = set()
            while of is not None and d["layers"][of].get("weights_of") is not None and of not in seen:
                seen.add(of)
                of = d["layers"][of]["weights_of"]
            if mlp and mlp["kind"] == "moe":
                r, x = mlp["router"], mlp["expert"]
                ex = Experts(r["experts"], r["top"], r.get("scale", 1.0), x.get("limit", 0.0), (mlp.get("shared") or {}).get("ff", 0))
                layers.append(LayerSpec(e["type"], e["mixer"], x["ff"], design.routing.act, ex, of))
            else:
                act = SILU if design.dense_act is None else design.dense_act
                layers.append(LayerSpec(e["type"], e["mixer"], mlp["ff"] if mlp else 0, act, None, of))
        lp = d.get("loop")
        return cls(name, d["width"], d["vocab"], layers, (lp["start"], lp["stop"], lp["times"]) if lp else None, d["norm"]["eps"],
                   design=design, streams=d.get("streams") or 0, embed_scale=(d.get("embedding") or {}).get("scale", 1.0),
                   residual_mult=d.get("residual_mult", 1.0), logit_scale=d.get("logit_scale", 1.0),
                   token_side=(d.get("token_side") or {}).get("dim", 0))

    @property
    def recurrent(self) -> bool:
        """Whether some layer's state cannot go back to an earlier position."""
        return any(p.mixer in RECURRENT for L in self.layers for _, p, _ in L.parts(self.design))

    def owner(self, i: int) -> int:
        """The layer whose parameters layer i uses."""
        of = self.layers[i].weights_of
        return i if of is None else of

    def layer_runs(self) -> list[int]:
        """Layers in the order they run."""
        n = len(self.layers)
        if not self.loop:
            return list(range(n))
        a, b, t = self.loop
        return list(range(a)) + list(range(a, b)) * t + list(range(b, n))

    def param_shapes(self) -> dict[str, tuple[int, ...]]:
        """Tensor names and shapes of a checkpoint (weights [out, in])."""
        W, D = self.hidden_size, self.design
        s = {"embed": (self.vocab_size, W), "final.norm": (W,)}
        if D.layer_norm:
            s["final.norm.b"] = (W,)
        if D.embed_norm:
            s["embed.norm"] = (W,)
        if not D.tied_head:
            s["head"] = (self.vocab_size, W)
        if self.loop and D.loop_input:
            s["loop.in"] = (W, 2 * W)
        if self.token_side:
            s["side.embed"] = (self.vocab_size, len(self.layers) * self.token_side)
        for i, L in enumerate(self.layers):
            if L.weights_of is not None:
                continue
            p = f"l{i}."
            if D.depth_average:
                s[p + "dwa"] = (i + 2,)
            if self.token_side:
                s[p + "side.gate"], s[p + "side.proj"], s[p + "side.norm"] = (self.token_side, W), (W, self.token_side), (W,)
            if L.mixer == "parallel" and D.beside_norms:
                s[p + "mix.left.out"] = s[p + "mix.right.out"] = (W,)
            for q in (1, 2) if L.ffn and not D.parallel_sublayers else (1,):
                s.update({p + n: (W,) for n in D.norms(q)})
                if self.streams:
                    s[p + f"hc{q}.in"] = s[p + f"hc{q}.out"] = (self.streams,)
                    s[p + f"hc{q}.mix"] = (self.streams, self.streams)
            if L.experts:
                s[p + "mlp.router"] = (L.experts.count, W)
                if D.routing.correction:
                    s[p + "mlp.correction"] = (L.experts.count,)
                units = {f"mlp.e{e}.": L.ffn for e in range(L.experts.count)} | ({"mlp.shared.": L.experts.shared} if L.experts.shared else {})
                for n, f in units.items():
                    s[p + n + "up"], s[p + n + "down"] = (f, W), (W, f)
                    if D.routing.gated:
                        s[p + n + "gate"] = (f, W)
            elif L.ffn:
                s[p + "mlp.up"], s[p + "mlp.down"] = (L.ffn, W), (W, L.ffn)
                if L.act == GELU1:
                    s[p + "mlp.up.b"], s[p + "mlp.down.b"] = (L.ffn,), (W,)
                elif L.act != RELU2:
                    s[p + "mlp.gate"] = (L.ffn, W)
            for side, part, traits in L.parts(D):
                self._mixer_shapes(s, p + "mix." + side, part, traits)
        return s

    def _mixer_shapes(self, s: dict, p: str, L: LayerSpec, traits: AttentionTraits):
        W, m = self.hidden_size, L.sizes
        if L.mixer == "rglru":
            n, b, taps = m["width"], m["blocks"], m["conv"]
            s[p + "y"] = s[p + "x"] = (n, W)
            s[p + "o"] = (W, n)
            s[p + "conv"] = (n, taps)
            s[p + "y.b"] = s[p + "x.b"] = s[p + "conv.b"] = s[p + "lam"] = (n,)
            s[p + "ra"] = s[p + "ri"] = (b, n // b, n // b)
            s[p + "ra.b"] = s[p + "ri.b"] = (b, n // b)
            return
        H, dv = m["heads"], m["vdim"]
        s[p + "o"] = (W, H * dv)
        if L.mixer == "attention":
            G, d = m["kv_heads"], m["dim"]
            s[p + "q"], s[p + "k"], s[p + "v"] = (H * d, W), (G * d, W), (G * dv, W)
            if traits.qk_norm == 1:
                s[p + "q.norm"], s[p + "k.norm"] = (H * d,), (G * d,)
            if traits.sink:
                s[p + "sink"] = (H,)
            if traits.gate or traits.wide_gate:
                s[p + "g"] = (H * dv if traits.wide_gate else H, W)
            if traits.dist_bias:
                s[p + "r1"] = s[p + "r2"] = (H,)
        elif L.mixer == "lightning":
            d = m["dim"]
            s[p + "q"] = s[p + "k"] = (H * d, W)
            s[p + "v"] = s[p + "g"] = (H * dv, W)
            s[p + "norm"] = (H * dv,)
        elif L.mixer == "latent_attention":
            d, r, R = m["dim"], m["rot_dim"], m["kv_rank"]
            s[p + "q"], s[p + "dkv"], s[p + "dkv.norm"] = (H * (d + r), W), (R + r, W), (R,)
            s[p + "uk"], s[p + "uv"] = (H * d, R), (H * dv, R)
        elif L.mixer == "gla":
            d, r = m["dim"], self.ranks[0]
            s[p + "q"] = s[p + "k"] = (H * d, W)
            s[p + "v"] = s[p + "g"] = (H * dv, W)
            s[p + "a1"], s[p + "a2"], s[p + "a2.b"] = (r, W), (H * d, r), (H * d,)
            s[p + "norm"] = (dv,)
        elif L.mixer in ("delta", "channel_delta"):
            K, d, taps = m["kv_heads"], m["dim"], m["conv"]
            for n, rows in (("q", K * d), ("k", K * d), ("v", H * dv)):
                s[p + n], s[p + n + ".conv"] = (rows, W), (rows, taps)
            s[p + "b"] = (H, W)
            s[p + "A_log"] = (H,)
            if L.mixer == "channel_delta":
                ra, rg = self.ranks
                s[p + "a1"], s[p + "a2"], s[p + "dt_bias"] = (ra, W), (H * d, ra), (H * d,)
                s[p + "g1"], s[p + "g2"] = (rg, W), (H * dv, rg)
            else:
                s[p + "a"] = (H, W)
                s[p + "g"] = (H * dv, W)
                s[p + "dt_bias"] = (H,)
            s[p + "norm"] = (dv,)
        else:
            N, G, taps = m["state"], m["groups"], m["conv"]
            ch = H * dv + 2 * G * N
            s[p + "in"], s[p + "conv"], s[p + "conv.b"] = (H * dv + ch + H, W), (ch, taps), (ch,)
            s[p + "A_log"] = s[p + "dt_bias"] = s[p + "D"] = (H,)
            s[p + "norm"] = (H * dv,)

    def synthetic(self, name: str) -> tuple[float, float]:
        """(mean, std) a synthetic checkpoint draws a tensor with: gains 1, slow decays, wide taps,
        streams that are read and written alike."""
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "A_log":
            return 0.5, 0.5
        if leaf == "dt_bias":
            return -3.0, 1.0
        if name.endswith("conv"):
            return 0.0, 0.4
        if name.endswith("conv.b"):
            return 0.0, 0.1
        if name.endswith("a2.b"):
            return 2.0, 1.5
        if leaf == "lam":
            return -3.0, 1.0
        if leaf in ("r1", "r2"):
            return (1.0 if leaf == "r1" else 0.3), 0.02
        if leaf == "dwa":
            return 1.0 / (int(name.split(".")[0][1:]) + 2), 0.1
        if leaf == "out":
            return 1.0, 0.0
        if name.endswith(".b") and not name.endswith(".mix.b"):
            return 0.0, 0.1
        if leaf in ("D", "norm", "norm1", "norm1b", "norm2", "norm2b"):
            plus_one = self.design.norm_plus_one and ".mix." not in name
            return 0.0 if plus_one else 1.0, 0.0
        if ".hc" in name:
            return {"in": 1.0, "out": 1.0, "mix": 0.0}[leaf] / self.streams, 0.5 / self.streams
        if leaf in ("correction", "sink"):
            return 0.0, 0.001 if leaf == "correction" else 1.0
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


def segedra_shape(name: str, width: int, heads: int, kv_heads: int, dim: int, window: int, experts: Experts, ff: int, dense_ff: int,
                  streams: int, vocab: int) -> LayeredConfig:
    """A Segedra-shaped model at a real model's widths, for measurements: a dense layer, then layers of
    experts, a loop over three of them, every third layer without a window."""
    def layer(i):
        m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "rot": {"base": 150000.0, "dims": dim},
             "mask": None if i % 3 == 2 else {"size": window}}
        return LayerSpec("attention", m, ff, BOUNDED, experts) if i else LayerSpec("attention", m, dense_ff, RELU2)
    return LayeredConfig(name, width, vocab, [layer(i) for i in range(8)], (1, 4, 2), 1e-5, design=DESIGNS["Segedra"], streams=streams,
                         embed_scale=width ** 0.5)


def regupel_shape(name: str, width: int, heads: int, kv_heads: int, dim: int, window: int, kept: int, experts: Experts, ff: int,
                  vocab: int) -> LayeredConfig:
    """A Regupel-shaped model at a real model's widths, for measurements: three of four layers carry windowed
    attention beside lightning attention (half the heads, values as wide as keys), every fourth is
    gated attention with a window four times as long; one of those uses another one's weights."""
    def layer(i):
        if i % 4 == 1:
            m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": 4 * window},
                 "rot": {"base": 500000.0, "dims": dim // 2, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
            return LayerSpec("attention", m, ff, SILU, experts, weights_of=1 if i == 5 else None)
        left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": window, "keep_first": kept}}
        n = heads // 2
        right = {"heads": n, "dim": dim, "vdim": dim, "decay": [1.0 - 2.0 ** -(1.0 + 9.0 * h / max(n - 1, 1)) for h in range(n)]}
        return LayerSpec("parallel", {"left": left, "right": right, "left_scale": 0.7, "right_scale": 0.7}, ff, SILU, experts)
    return LayeredConfig(name, width, vocab, [layer(i) for i in range(8)], None, 1e-6, design=DESIGNS["Regupel"], embed_scale=width ** 0.5,
                         residual_mult=0.8, logit_scale=0.25)


def kivorax_shape(name: str, width: int, heads: int, kv_heads: int, dim: int, experts: Experts, ff: int, dense_ff: int, side: int, vocab: int,
                  rank: int = 128, key: int = 128) -> LayeredConfig:
    """A Kivorax-shaped model at a real model's widths, for measurements: a dense layer, then layers of experts;
    half of the mixers are delta rules with key x key states, a quarter gated linear attention with
    key / 2 x key states, a quarter attention beside a recurrent block as wide as the model."""
    n = width // key
    dlt = ("channel_delta", {"heads": n, "kv_heads": n, "dim": key, "vdim": key, "conv": 4})
    lin = ("gla", {"heads": n, "dim": key // 2, "vdim": key, "tau": 16.0})
    two = ("parallel", {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "q_temp": {"coef": 0.1, "every": 1024}},
                        "right": {"width": width, "blocks": n, "conv": 4}})
    order = [dlt, lin, dlt, two] * 2
    layers = [LayerSpec(m, s, ff, RELU2, experts) if i else LayerSpec(m, s, dense_ff, GELU1) for i, (m, s) in enumerate(order)]
    return LayeredConfig(name, width, vocab, layers, None, 1e-5, design=DESIGNS["Kivorax"], embed_scale=width ** 0.5, token_side=side,
                         ranks=(rank, rank))


KIVORAX_W1024 = kivorax_shape("kivorax-w1024-shape", 1024, 16, 4, 64, Experts(32, 4), 512, 4096, 128, 32000)
KIVORAX_W2048 = kivorax_shape("kivorax-w2048-shape", 2048, 32, 4, 128, Experts(128, 8), 768, 8192, 256, 151936)
KIVORAX_W3072 = kivorax_shape("kivorax-w3072-shape", 3072, 64, 8, 64, Experts(32, 4), 3072, 12288, 256, 201088)
REGUPEL_W1024 = regupel_shape("regupel-w1024-shape", 1024, 16, 4, 64, 128, 16, Experts(32, 4, shared=512), 512, 32000)
REGUPEL_W2048 = regupel_shape("regupel-w2048-shape", 2048, 32, 4, 128, 512, 64, Experts(128, 8, shared=768), 768, 151936)
REGUPEL_W2880 = regupel_shape("regupel-w2880-shape", 2880, 64, 8, 64, 128, 128, Experts(32, 4, shared=2880), 2880, 201088)
SEGEDRA_W1024 = segedra_shape("segedra-w1024-shape", 1024, 16, 4, 64, 128, Experts(32, 4, 1.0, 7.0), 512, 4096, 2, 32000)
SEGEDRA_W2048 = segedra_shape("segedra-w2048-shape", 2048, 32, 4, 128, 512, Experts(128, 8, 2.5, 7.0), 768, 8192, 4, 151936)
SEGEDRA_W2880 = segedra_shape("segedra-w2880-shape", 2880, 64, 8, 64, 128, Experts(32, 4, 1.0, 7.0), 2880, 11520, 4, 201088)
RALAPEL_W1024 = bench_shape("ralapel-w1024-shape", 1024, 4096, 32000)
RALAPEL_W2048 = bench_shape("ralapel-w2048-shape", 2048, 8192, 128256)
RALAPEL_W4096 = bench_shape("ralapel-w4096-shape", 4096, 14336, 128256)
