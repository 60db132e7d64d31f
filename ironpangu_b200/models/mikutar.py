"""Mikutar: a decoder of parallel layers - mixer and feed-forward read one norm, x += mixer(h) + ff(h) with h = rms(x) w1 - over an f32
residual, some of whose layers run several times in a row; the embedding table is the output matrix.

  attention     grouped heads over the last ``mask.size`` positions; biases on q, k and the output; q and k normed over all their heads
                together; interleaved rotation of the first ``rot.dims`` columns; the values are the keys as projected
  attention_2   grouped heads over the query's own stretch of ``mask.size`` positions; scores softly capped, then less a slope per head
                times the distance; no rotation
  both          head h times sigmoid(W_g h)_h; W_o
  dense         W_down (relu(W_gate h) (W_up h))
  moe           sigmoid scores; chosen by score + correction among the best groups, weighted by the score; limited units g' sigmoid(1.702 g')
                (u' + 1); a shared expert for every row
  loop          layers start .. stop - 1 run ``times`` times with the same weights, each pass with pages of its own; before each pass but
                the first the embedding output joins the residual

What every row takes of a feed-forward (a dense one, the shared expert) and the mixer end in ONE matrix product: their operands lie side by
side in a row, W_o beside W_down. ``MikutarDecoder`` and ``MikutarRows`` are the decode and packed-step executors (``stream_decoder.py``).
In bf16 the linears take bf16 operands with f32 accumulation; norms, rotations, scores, weights, the router and the residual are f32. With
``dtype=torch.float32`` every product is a true f32 FMA.

A checkpoint directory is ``config.json`` (``"architecture": "Mikutar"``) + safetensors; see :func:`weight_shapes` for the names."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..ops import parallel_layer as PL
from ..ops import stream_norm as N
from ..ops.linear_attn import DevicePlan, RotaryTables
from ..ops.routed_experts import ExpertBuffers, ExpertsShape, RoutedExperts
from ..ops.window_attn import GroupedAttention, GroupedBuffers, GroupedShape
from ..parallel.fabric import Fabric
from . import checkpoint
from .checkpoint import pad8
from .stream_decoder import ATTN_ROWS, BF16, F32, StreamDecoder, StreamRows

KERNEL_UNITS = ("misc", "post_norm", "linear_f32", "window_attn", "decode_gqa", "fa_prefill", "moe_rows", "moe_prefill", "tc_grouped", "decode_post_norm", "decode_moe",
                "sampling", "tc_gemm", "tc_gemm_2sm")
MIXERS = ("attention", "attention_2")
ALPHA = 1.702              # of the limited units


# ---------------------------------------------------------------------------------------------------------------------------
# configuration
# ---------------------------------------------------------------------------------------------------------------------------
@dataclass
class LayerConfig:
    kind: str
    mixer: GroupedShape
    ff: int = 0                                  # width of the unit every row takes: the dense feed-forward or the shared expert (0: none)
    unit: N.GatedUnit = N.GatedUnit("relu")
    experts: Optional[ExpertsShape] = None       # routed experts beside it


@dataclass
class LoopConfig:
    start: int = 0
    stop: int = 0
    times: int = 1


@dataclass
class MikutarConfig:
    vocab: int
    width: int
    eps: float
    logit_cap: float = 0.0
    layers: List[LayerConfig] = field(default_factory=list)
    loop: LoopConfig = field(default_factory=LoopConfig)
    page_tokens: int = 16

    @staticmethod
    def from_dict(j: dict) -> "MikutarConfig":
        if j.get("architecture") != "Mikutar":
            raise ValueError(f"not a Mikutar configuration (architecture {j.get('architecture')!r})")
        width, layers = int(j["width"]), []
        for i, e in enumerate(j["layers"]):
            m, f, kind = e["mixer"], e.get("mlp"), e["type"]
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            sizes = dict(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                         window=int((m.get("mask") or {}).get("size", 0)))
            if kind == "attention":
                rot = m.get("rot") or {}
                mixer = GroupedShape(**sizes, rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)), norm=True, keys_are_values=True, bias=True)
            else:
                mixer = GroupedShape(**sizes, chunked=True, cap=float(m.get("softcap") or 0.0), biased=True)
            layer = LayerConfig(kind, mixer)
            if f is not None and f.get("kind") == "dense":
                layer.ff = int(f["ff"])
            elif f is not None and f.get("kind") == "moe":
                limited = lambda limit: N.GatedUnit("limited", float(limit), ALPHA)
                r, shared = f["router"], f.get("shared")
                groups = r.get("groups") or {"count": 1, "keep": 1}
                layer.experts = ExpertsShape(width, int(r["experts"]), int(r["top"]), int(f["expert"]["ff"]), scoring="sigmoid", renorm=False,
                                             groups=int(groups["count"]), keep=int(groups["keep"]), unit=limited(f["expert"]["limit"]))
                if shared:
                    layer.ff, layer.unit = int(shared["ff"]), limited(shared["limit"])
            elif f is not None:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
            layers.append(layer)
        loop = j.get("loop") or {}
        return MikutarConfig(int(j["vocab"]), width, float(j["norm"]["eps"]), float(j.get("logit_softcap") or 0.0), layers,
                             LoopConfig(int(loop.get("start", 0)), int(loop.get("stop", 0)), int(loop.get("times", 1)))).validate()

    def to_dict(self) -> dict:
        out = []
        for l in self.layers:
            m, x = l.mixer, l.experts
            d = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "mask": {"size": m.window}}
            if l.kind == "attention":
                d["rot"] = {"dims": m.rot_dims, "base": m.rot_base}
            else:
                d["softcap"] = m.cap
            f = None
            if x is not None:
                f = {"kind": "moe", "expert": {"ff": x.ff, "limit": x.unit.limit}, "router": {"experts": x.experts, "top": x.top, "groups": {"count": x.groups, "keep": x.keep}}}
                if l.ff:
                    f["shared"] = {"ff": l.ff, "limit": l.unit.limit}
            elif l.ff:
                f = {"kind": "dense", "ff": l.ff}
            out.append({"type": l.kind, "mixer": d, "mlp": f})
        return {"architecture": "Mikutar", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "logit_softcap": self.logit_cap, "layers": out,
                "loop": {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}}

    def validate(self) -> "MikutarConfig":
        if not self.layers:
            raise ValueError("no layers")
        o = self.loop
        if not 0 <= o.start <= o.stop <= len(self.layers) or o.times < 1:
            raise ValueError(f"loop over layers {o.start} .. {o.stop - 1}, {o.times} times, of {len(self.layers)}")
        if self.logit_cap < 0:
            raise ValueError("the cap of the logits must not be negative")
        for i, l in enumerate(self.layers):
            try:
                l.mixer.check()
                l.unit.check()
                if l.ff < 0:
                    raise ValueError("negative feed-forward width")
                if l.experts is not None:
                    l.experts.check()
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
        return self

    def order(self) -> List[tuple]:
        """``(layer, whether the embedding output joins the residual first)`` of every layer run."""
        o, n = self.loop, len(self.layers)
        stop = min(o.stop, n)
        head, tail = range(min(o.start, n)), range(stop, n) if stop > o.start else range(min(o.start, n), n)
        body = [(i, t > 0 and i == o.start) for t in range(o.times) for i in range(o.start, stop)]
        return [(i, False) for i in head] + body + [(i, False) for i in tail]

    @property
    def window(self) -> int:
        """How far back any layer sees when every layer has a limit, else 0."""
        w = [l.mixer.window for l in self.layers]
        return max(w) if all(w) else 0

    def param_count(self) -> int:
        return checkpoint.param_count(weight_shapes(self))

    def active_params(self) -> int:
        """Parameters a token uses, counting looped layers once: all but the experts it does not choose."""
        return self.param_count() - sum((l.experts.experts - l.experts.top) * 3 * l.experts.ff * self.width for l in self.layers if l.experts)

    @staticmethod
    def tiny() -> "MikutarConfig":
        """Both mixers in unequal sizes, every feed-forward, a layer without one, a loop; odd sizes."""
        a = GroupedShape(6, 2, 40, 40, 0.2, 24, rot_dims=24, rot_base=1e5, norm=True, keys_are_values=True, bias=True)
        b = GroupedShape(3, 3, 24, 56, 0.3, 20, chunked=True, cap=9.0, biased=True)
        limited = lambda v: N.GatedUnit("limited", v, ALPHA)
        x = ExpertsShape(136, 12, 3, 40, scoring="sigmoid", renorm=False, groups=3, keep=2, unit=limited(1.5))
        y = ExpertsShape(136, 5, 2, 24, scoring="sigmoid", renorm=False, unit=limited(0.7))
        return MikutarConfig(384, 136, 1e-5, 25.0, [LayerConfig("attention", a, 200), LayerConfig("attention_2", b, 72, limited(2.5), x), LayerConfig("attention", a),
                                                    LayerConfig("attention_2", b, experts=y)], LoopConfig(1, 3, 2)).validate()

    @staticmethod
    def text(layers: int = 16, width: int = 2048, heads: int = 16, kv_heads: int = 4, dim: int = 128, ff: int = 6144, experts: int = 64, top: int = 8, expert_ff: int = 768,
             shared_ff: int = 768, vocab: int = 128000, window: int = 1024, chunk: int = 2048, loop: tuple = (0, 0, 1)) -> "MikutarConfig":
        """Dense and routed feed-forwards in turn, every fourth layer chunked."""
        a = GroupedShape(heads, kv_heads, dim, dim, dim ** -0.5, window, rot_dims=dim, rot_base=5e5, norm=True, keys_are_values=True, bias=True)
        b = GroupedShape(heads, kv_heads, dim, dim, dim ** -0.5, chunk, chunked=True, cap=20.0, biased=True)
        limited = N.GatedUnit("limited", 7.0, ALPHA)
        x = ExpertsShape(width, experts, top, expert_ff, scoring="sigmoid", renorm=False, groups=max(1, experts // 16), keep=max(1, experts // 32), unit=limited)
        out = []
        for i in range(layers):
            l = LayerConfig(*(("attention_2", b) if i % 4 == 3 else ("attention", a)))
            if i % 2:
                l.ff, l.unit, l.experts = shared_ff, limited, x
            else:
                l.ff = ff
            out.append(l)
        return MikutarConfig(vocab, width, 1e-6, 30.0, out, LoopConfig(*loop)).validate()


PRESETS = {"mikutar-tiny": MikutarConfig.tiny, "mikutar-text": MikutarConfig.text}


# ---------------------------------------------------------------------------------------------------------------------------
# weights
# ---------------------------------------------------------------------------------------------------------------------------
def weight_shapes(c: MikutarConfig) -> Dict[str, tuple]:
    """Checkpoint tensor names -> shapes (bf16 in the file)."""
    s = {"embed": (c.vocab, c.width)}
    for i, l in enumerate(c.layers):
        p, m, x = f"l{i}.", l.mixer, l.experts
        q, k, v = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
        s.update({p + "norm1": (c.width,), p + "mix.q": (q, c.width), p + "mix.k": (k, c.width), p + "mix.g": (m.heads, c.width), p + "mix.o": (c.width, m.heads * m.vdim)})
        if not m.keys_are_values:
            s[p + "mix.v"] = (v, c.width)
        if m.bias:
            s.update({p + "mix.q.b": (q,), p + "mix.k.b": (k,), p + "mix.o.b": (c.width,)})
        if m.norm:
            s.update({p + "mix.q.norm": (q,), p + "mix.k.norm": (k,)})
        units = [(f"e{e}.", x.ff) for e in range(x.experts)] if x else []
        if x:
            s.update({p + "mlp.router": (x.experts, c.width), p + "mlp.correction": (x.experts,)})
        if l.ff:
            units.append(("shared." if x else "", l.ff))
        for name, ff in units:
            n = p + "mlp." + name
            s.update({n + "gate": (ff, c.width), n + "up": (ff, c.width), n + "down": (c.width, ff)})
    s["final.norm"] = (c.width,)
    return s


def random_weights(c: MikutarConfig, device, seed: int = 0, std: float = 0.02) -> Dict[str, torch.Tensor]:
    """Random-init checkpoint tensors: N(0, std) matrices, biases and corrections, gains 1 + N(0, std)."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in weight_shapes(c).items():
        t = torch.empty(shape, dtype=BF16, device=device).normal_(0.0, std, generator=g)
        out[name] = t + 1.0 if "norm" in name else t
    return out


def save_checkpoint(path, c: MikutarConfig, weights: Dict[str, torch.Tensor]) -> None:
    checkpoint.save(path, c, weights)


def load_checkpoint(path) -> tuple:
    """``(config, weights on the host)`` of a checkpoint directory; every expected tensor must be there with its shape."""
    return checkpoint.load(path, MikutarConfig.from_dict, weight_shapes)


# ---------------------------------------------------------------------------------------------------------------------------
# executors
# ---------------------------------------------------------------------------------------------------------------------------
class _Rows:
    """Step buffers for up to ``rows`` rows (leading dimensions padded to 8 elements, padding zero)."""

    def __init__(self, dec: "MikutarDecoder", rows: int, chunked: bool):
        c, dev, A = dec.cfg, dec.fabric.device, dec.dtype
        z = lambda n, dt=A: torch.zeros(rows, pad8(n), dtype=dt, device=dev)
        self.rows = rows
        self.x, self.x2 = z(c.width, F32), z(c.width, F32)           # residual stream (two: fused prologues write the other one)
        self.first = z(c.width, F32) if any(add for _, add in c.order()) else None      # the embedding output
        self.xa, self.y = z(c.width), z(c.width, F32)
        shapes = [l.mixer for l in c.layers]
        self.attn = GroupedBuffers(shapes, rows, A, dev, chunked=chunked, max_context=dec.max_context, group=ATTN_ROWS)
        self.join = PL.JoinBuffers([L["join"] for L in dec.layers], rows, A, dev)
        routed = [l.experts for l in c.layers if l.experts is not None]
        self.experts = ExpertBuffers(routed, rows, A, dev) if routed else None
        self.rotary = RotaryTables([(m.rot_dims, m.rot_base) for m in shapes], rows, dev)


class MikutarDecoder(StreamDecoder):
    """Decode executor: see :class:`StreamDecoder`. ``layers`` holds the weights, ``runs`` the layer runs with their pages."""

    name = "mikutar"

    def make_rows(self, rows: int, chunked: bool) -> _Rows:
        return _Rows(self, rows, chunked)

    def _load(self, W: Dict[str, torch.Tensor]) -> None:
        c, dev = self.cfg, self.fabric.device
        self.embed = self.head = self._mat(W, "embed")
        self.final_norm, self.logit_cap = self._vec(W, "final.norm"), c.logit_cap
        self.layers: List[dict] = []
        for i, l in enumerate(c.layers):
            p = f"l{i}."
            unit = PL.UnitWeights(W, p + "mlp." + ("shared." if l.experts else ""), l.ff, l.unit, dev, self.dtype) if l.ff else None
            self.layers.append({
                "norm1": self._vec(W, p + "norm1"), "mix": GroupedAttention(l.mixer, W, p + "mix.", dev, self.dtype),
                "join": PL.Join(W[p + "mix.o"], W.get(p + "mix.o.b"), unit, dev, self.dtype),
                "experts": RoutedExperts(l.experts, W, p + "mlp.", dev, self.dtype, bias="correction") if l.experts else None})
        self.fused = self.dtype == BF16 and c.width % 8 == 0         # the fused decode chain norms unpadded rows

    def _state_bytes(self) -> tuple:
        es = torch.empty((), dtype=self.dtype).element_size()
        return sum(self.cfg.layers[i].mixer.row for i, _ in self.cfg.order()) * es, 0

    def _make_states(self) -> None:
        self.runs = [dict(self.layers[i], add=add, pages=self.layers[i]["mix"].make_pages(self.num_pages, self.cfg.page_tokens, self.fabric.device, self.dtype))
                     for i, add in self.cfg.order()]

    @classmethod
    def from_checkpoint(cls, path, fabric: Fabric, **kw) -> "MikutarDecoder":
        c, w = load_checkpoint(path)
        return cls(c, w, fabric, **kw)

    # -- layers ------------------------------------------------------------------------------------------------------------
    def _attend(self, B: _Rows, R: dict, m: int, pos, slot, plan: Optional[DevicePlan]) -> None:
        s = R["mix"].shape
        R["mix"].attend(B.attn, m, R["pages"], B.rotary.get(s.rot_dims, s.rot_base), pos, slot, plan, self.page_table, self.cfg.eps, R["join"].operand(B.join, m),
                        self.fabric.desc.status)

    def _layers(self, B: _Rows, m: int, tok, pos, slot, plan: Optional[DevicePlan], final: bool, probe: Optional[list] = None) -> None:
        """All layer runs over ``m`` rows as separate row operators and matrix products; the residual ends in ``B.x``, and with ``final`` the
        normalised rows for the output matrix in ``B.xa``."""
        c, st, W = self.cfg, self.fabric.desc.status, self.cfg.width
        x, xa = B.x[:m, :W], B.xa[:m]
        first = None if B.first is None else B.first[:m, :W]
        N.embed_rows(tok, self.embed, x, xa, gain=self.runs[0]["norm1"], eps=c.eps, copy=first, status_ptr=st)
        B.rotary.fill(pos)
        if B.experts is not None:
            B.experts.start(m)
        for i, R in enumerate(self.runs):
            nxt = self.runs[i + 1] if i + 1 < len(self.runs) else None
            gain = nxt["norm1"] if nxt else self.final_norm if final else None
            extra = first if nxt and nxt["add"] else None
            R["mix"].project(B.attn, xa, st)
            R["join"].unit_rows(B.join, xa, st)
            self._attend(B, R, m, pos, slot, plan)
            y = R["join"].rows(B.join, m, B.y[:m], st)
            then = (None, None) if probe is not None else (gain, extra)
            if R["experts"] is not None:
                R["experts"].rows(B.experts, m, xa, None, then[0], c.eps, B.x[:m], st, base=y, extra=None if then[1] is None else B.first[:m])
            else:
                N.post_norm_add(y[..., :W], None, c.eps, x, xa, *then)
            if probe is not None:                  # the residual as the layer leaves it; what comes before the next one follows
                probe.append(x.clone())
                N.post_norm_add(None, None, c.eps, x, xa, gain, extra)

    def _layers_fused(self, B: _Rows, n: int, tok, pos, slot) -> None:
        """Decode rows: residual update, norm, projection, the unit every row takes and the router in one launch at the front of a layer, one
        product at its end. Ends like :meth:`_layers` with ``final``."""
        c, st = self.cfg, self.fabric.desc.status
        x, x2, xa, y = B.x[:n], B.x2[:n], B.xa[:n], B.y[:n]
        first = None if B.first is None else B.first[:n]
        N.embed_rows(tok, self.embed, x, xa, copy=first, status_ptr=st)
        B.rotary.fill(pos)
        owed = None                            # sublayer outputs that the residual still lacks
        for R in self.runs:
            join, experts = R["join"], R["experts"]
            PL.parallel_in(owed, first if R["add"] else None, R["norm1"], c.eps, x, x2, xa, R["mix"], B.attn.proj[:n], join, B.join, experts, B.experts,
                           self.fabric.ticket_ptr)
            x, x2 = x2, x
            if experts is not None:
                experts.decode_chosen(B.experts, n, xa, y)
            self._attend(B, R, n, pos, slot, None)
            join.decode(B.join, n, y, y if experts is not None else None)
            owed = y
        N.post_norm_add(y, None, c.eps, x, xa, self.final_norm)


class MikutarRows(StreamRows):
    """Packed-step executor: see :class:`StreamRows`."""
