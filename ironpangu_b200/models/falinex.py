"""Falinex: a decoder whose layers mix by retention, lightning attention or sliding-window attention in any order, with the norm on
every sublayer's OUTPUT (x += rms(sublayer(x)) * w) over an f32 residual stream, and dense GELU feed-forwards. Layers may share
another layer's weights (``weights_of``) with a state or cache of their own.

  retention     q, k rotated (half layout), k * dim^-1/2; S = decay S + k v^T, o = S^T q (f32 state); o / rms per head;
                * silu(W_g x); W_o
  lightning     q, k, v through SiLU; the same recurrence without rotation or scale; rms over all heads together with a gain;
                * sigmoid(W_g x); W_o
  attention     grouped heads; rms of q and k per head with a gain; interleaved rotation; scores * scale over the last ``mask.size``
                positions; softmax with a learned sink per head in the denominator; * sigmoid(W_g x); W_o

``FalinexDecoder`` and ``FalinexRows`` are the decode and packed-step executors (``stream_decoder.py``).
In bf16 the linears take bf16 operands with f32 accumulation; norms, rotations, scores, recurrences and the residual are f32.
With ``dtype=torch.float32`` every product is a true f32 FMA.

A checkpoint directory is ``config.json`` (``"architecture": "Falinex"``) + safetensors; see :func:`weight_shapes` for the names."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..ops import stream_norm as N
from ..ops import window_attn as WA
from ..ops.linear_attn import CHUNK, TILE, DecayedMixer, DevicePlan, RotaryTables
from ..parallel.fabric import Fabric
from . import checkpoint
from .checkpoint import pad8
from .stream_decoder import ATTN_ROWS, BF16, F32, StreamDecoder, StreamRows

KERNEL_UNITS = ("misc", "post_norm", "linear_f32", "linear_attn", "linear_attn_tc", "window_attn", "decode_post_norm", "decode_gqa", "fa_prefill", "decode_moe", "sampling",
                "tc_gemm", "tc_gemm_2sm")


# ---------------------------------------------------------------------------------------------------------------------------
# configuration
# ---------------------------------------------------------------------------------------------------------------------------
@dataclass
class MixerConfig:
    kind: str                          # retention | lightning | attention
    heads: int
    dim: int
    vdim: int
    kv_heads: int = 0                  # attention
    decay: tuple = ()                  # retention, lightning
    rot_dims: int = 0
    rot_base: float = 10000.0
    window: int = 0                    # attention: 0 = no window
    scale: float = 1.0                 # attention

    @property
    def recurrent(self) -> bool:
        return self.kind != "attention"

    @property
    def qk_groups(self) -> int:
        return self.heads if self.recurrent else self.kv_heads

    @property
    def q_shape(self) -> tuple:
        """(heads, columns from one query head to the next, columns of a head)."""
        return self.heads, WA.tile_width(self.dim) if self.tiles else self.dim, self.dim

    @property
    def tiles(self) -> bool:
        """Attention whose heads fit the tiles of the tensor-core kernel."""
        return not self.recurrent and max(self.dim, self.vdim) <= 128

    @property
    def ctx_shape(self) -> tuple:
        return self.kv_heads, self.q_shape[1]

    @property
    def splits(self) -> int:
        return WA.split_form(self.heads, self.kv_heads, self.dim, self.vdim, self.window) if not self.recurrent and self.q_shape[1] == self.dim else 0

    @property
    def columns(self) -> List[int]:
        """Widths of q, k, v and the gate in the packed input projection."""
        return [self.heads * self.dim, self.qk_groups * self.dim, self.qk_groups * self.vdim, self.heads * self.vdim]


@dataclass
class LayerConfig:
    mixer: MixerConfig
    ff: int = 0                        # 0: no feed-forward
    weights_of: Optional[int] = None


@dataclass
class FalinexConfig:
    vocab: int
    width: int
    eps: float
    layers: List[LayerConfig] = field(default_factory=list)
    page_tokens: int = 16

    @staticmethod
    def from_dict(j: dict) -> "FalinexConfig":
        if j.get("architecture") != "Falinex":
            raise ValueError(f"not a Falinex configuration (architecture {j.get('architecture')!r})")
        layers = []
        for i, e in enumerate(j["layers"]):
            m, kind = e["mixer"], e["type"]
            if kind not in ("retention", "lightning", "attention"):
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            mask = m.get("mask") or {}
            rot = m.get("rot") or {}
            mc = MixerConfig(kind, int(m["heads"]), int(m["dim"]), int(m["vdim"]), kv_heads=int(m.get("kv_heads", m["heads"])) if kind == "attention" else 0,
                             decay=tuple(float(d) for d in m.get("decay", ())), rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)),
                             window=int(mask.get("size", 0)), scale=float(m.get("scale", 1.0)))
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(LayerConfig(mc, int(mlp["ff"]) if mlp is not None else 0, e.get("weights_of")))
        return FalinexConfig(int(j["vocab"]), int(j["width"]), float(j["norm"]["eps"]), layers).validate()

    def to_dict(self) -> dict:
        out = []
        for l in self.layers:
            m = l.mixer
            d = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
            if m.recurrent:
                d["decay"] = list(m.decay)
            else:
                d.update(kv_heads=m.kv_heads, mask={"size": m.window}, scale=m.scale)
            if m.rot_dims:
                d["rot"] = {"base": m.rot_base, "dims": m.rot_dims}
            e = {"type": m.kind, "mixer": d, "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None}
            if l.weights_of is not None:
                e["weights_of"] = l.weights_of
            out.append(e)
        return {"architecture": "Falinex", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": out}

    def validate(self) -> "FalinexConfig":
        for i, l in enumerate(self.layers):
            m = l.mixer
            if m.rot_dims % 2 or m.rot_dims > m.dim:
                raise ValueError(f"layer {i}: rotation of {m.rot_dims} columns in heads of {m.dim}")
            if m.recurrent and len(m.decay) != m.heads:
                raise ValueError(f"layer {i}: {m.heads} heads but {len(m.decay)} decay factors")
            if not m.recurrent and (m.kv_heads < 1 or m.heads % m.kv_heads or max(m.dim, m.vdim) > 256):
                raise ValueError(f"layer {i}: attention heads {m.heads} / {m.kv_heads} of {m.dim} / {m.vdim} columns are not supported")
            if l.weights_of is not None:
                j = self.owner(i)
                if (self.layers[j].mixer, self.layers[j].ff) != (m, l.ff):
                    raise ValueError(f"layer {i} shares the weights of layer {j} but not its sizes")
        return self

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen or not 0 <= self.layers[i].weights_of < len(self.layers):
                raise ValueError(f"layer {i}: weights_of does not lead to a layer with weights")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    @property
    def window(self) -> int:
        """The longest window when every attention layer has one, else 0."""
        w = [l.mixer.window for l in self.layers if not l.mixer.recurrent]
        return max(w) if w and all(w) else 0

    def param_count(self) -> int:
        return checkpoint.param_count(weight_shapes(self))

    @staticmethod
    def tiny() -> "FalinexConfig":
        """Every mixer, a shared layer, a layer without a feed-forward; odd sizes."""
        ret = MixerConfig("retention", 3, 24, 40, decay=(0.9, 0.98, 0.995), rot_dims=16, rot_base=1e4)
        lig = MixerConfig("lightning", 2, 32, 24, decay=(0.8, 0.99))
        att = MixerConfig("attention", 6, 40, 32, kv_heads=2, rot_dims=24, rot_base=1e5, window=24, scale=0.2)
        return FalinexConfig(384, 128, 1e-5, [LayerConfig(att, 192), LayerConfig(ret, 0), LayerConfig(lig, 192), LayerConfig(att, 192, 0)]).validate()

    @staticmethod
    def text2b(layers: int = 24, width: int = 2048, heads: int = 16, kv_heads: int = 4, dim: int = 128, ff: int = 6144, vocab: int = 151936,
               window: int = 1024) -> "FalinexConfig":
        """A 2B-class stack: (lightning, retention, retention, attention) repeated."""
        dec = lambda lo: tuple(1.0 - 2.0 ** -(lo + 6.0 * h / max(1, heads - 1)) for h in range(heads))
        lig = MixerConfig("lightning", heads, dim, dim, decay=dec(2.0))
        ret = MixerConfig("retention", heads, dim, dim, decay=dec(5.0), rot_dims=dim, rot_base=1e4)
        att = MixerConfig("attention", heads, dim, dim, kv_heads=kv_heads, rot_dims=dim, rot_base=1e6, window=window, scale=dim ** -0.5)
        return FalinexConfig(vocab, width, 1e-5, [LayerConfig((lig, ret, ret, att)[i % 4], ff) for i in range(layers)]).validate()


PRESETS = {"falinex-tiny": FalinexConfig.tiny, "falinex2b": FalinexConfig.text2b}


# ---------------------------------------------------------------------------------------------------------------------------
# weights
# ---------------------------------------------------------------------------------------------------------------------------
def weight_shapes(c: FalinexConfig) -> Dict[str, tuple]:
    """Checkpoint tensor names -> shapes (bf16 in the file)."""
    s = {"embed": (c.vocab, c.width), "final.norm": (c.width,), "head": (c.vocab, c.width)}
    for i, l in enumerate(c.layers):
        if l.weights_of is not None:
            continue
        p, m = f"l{i}.", l.mixer
        q, k, v, g = m.columns
        s[p + "norm1"] = (c.width,)
        s.update({p + "mix.q": (q, c.width), p + "mix.k": (k, c.width), p + "mix.v": (v, c.width), p + "mix.g": (g, c.width), p + "mix.o": (c.width, g)})
        if m.kind == "lightning":
            s[p + "mix.norm"] = (g,)
        if m.kind == "attention":
            s.update({p + "mix.q.norm": (m.dim,), p + "mix.k.norm": (m.dim,), p + "mix.sink": (m.heads,)})
        if l.ff:
            s.update({p + "norm2": (c.width,), p + "mlp.up": (l.ff, c.width), p + "mlp.down": (c.width, l.ff)})
    return s


def random_weights(c: FalinexConfig, device, seed: int = 0, std: float = 0.02) -> Dict[str, torch.Tensor]:
    """Random-init checkpoint tensors: N(0, std) matrices, gains 1 + N(0, std), sinks N(0, 1)."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in weight_shapes(c).items():
        t = torch.empty(shape, dtype=BF16, device=device).normal_(0.0, 1.0 if name.endswith("sink") else std, generator=g)
        out[name] = t + 1.0 if "norm" in name else t
    return out


def save_checkpoint(path, c: FalinexConfig, weights: Dict[str, torch.Tensor]) -> None:
    """Write ``config.json`` and ``model.safetensors`` (bf16)."""
    checkpoint.save(path, c, weights)


def load_checkpoint(path) -> tuple:
    """``(config, weights on the host)`` of a checkpoint directory; every expected tensor must be there with its shape."""
    return checkpoint.load(path, FalinexConfig.from_dict, weight_shapes)


# ---------------------------------------------------------------------------------------------------------------------------
# executors
# ---------------------------------------------------------------------------------------------------------------------------
class _Rows:
    """Step buffers for up to ``rows`` rows (leading dimensions padded to 8 elements, padding zero)."""

    def __init__(self, dec: "FalinexDecoder", rows: int, chunked: bool):
        c, dev, A = dec.cfg, dec.fabric.device, dec.dtype
        mix = [l.mixer for l in c.layers]
        z = lambda n, dt=A: torch.zeros(rows, pad8(n), dtype=dt, device=dev)
        self.rows = rows
        self.x, self.x2 = z(c.width, F32), z(c.width, F32)           # residual stream (two: fused prologues write the other one)
        self.xa, self.y = z(c.width), z(c.width, F32)
        self.proj = z(max(sum(m.columns) for m in mix))
        self.o = z(max([m.heads * m.vdim for m in mix if m.recurrent] or [1]), F32)
        att = [m for m in mix if not m.recurrent]
        # queries at the stride of the tensor-core tiles where they have one (padding columns stay zero: one buffer per shape)
        self.q = {m.q_shape: torch.zeros(rows, m.heads * m.q_shape[1], dtype=A, device=dev) for m in att}
        splits = [m.heads * m.splits * (m.vdim + 2) for m in att if m.splits]
        self.split_scratch = torch.empty(min(rows, ATTN_ROWS) * max(splits), dtype=F32, device=dev) if splits and A == BF16 else None
        self.ctx = {}
        if chunked and A == BF16:
            for m in att:
                if m.tiles:
                    cap = WA.context_rows(rows, m.window) if m.window else (dec.max_context + 31) // 32 * 32
                    k0, v0 = self.ctx.get(m.ctx_shape, (None, None))
                    if k0 is None or k0.shape[0] < cap:
                        self.ctx[m.ctx_shape] = (torch.zeros(cap, m.kv_heads * m.q_shape[1], dtype=A, device=dev),
                                                 torch.zeros(m.kv_heads * 128, cap, dtype=A, device=dev))
        self.mixed = {w: z(w) for w in {m.heads * m.vdim for m in mix}}      # one per width: the padding columns must stay zero
        self.act = {w: z(w) for w in {l.ff for l in c.layers if l.ff}}
        self.rotary = RotaryTables([(m.rot_dims, m.rot_base) for m in mix], rows, dev)
        self.scratch = None
        rec = [m for m in mix if m.recurrent]
        if chunked and rec:
            f = lambda n: torch.empty(n, dtype=F32, device=dev)
            nch = rows // dec.chunk + dec.num_slots + 1              # chunks of a step: whole ones and one ragged end per sequence
            wide = 0 if dec.tensor_recurrence else rows              # rows of q, k, v of the f32 form
            self.scratch = (f(wide * max(m.heads * m.dim for m in rec)), f(wide * max(m.heads * m.dim for m in rec)),
                            f(wide * max(m.heads * m.vdim for m in rec)), f(nch * max(m.heads * m.dim * m.vdim for m in rec)))


class FalinexDecoder(StreamDecoder):
    """Decode executor: see :class:`StreamDecoder`."""

    name = "falinex"

    def make_rows(self, rows: int, chunked: bool) -> _Rows:
        return _Rows(self, rows, chunked)

    def _load(self, W: Dict[str, torch.Tensor]) -> None:
        c, dev = self.cfg, self.fabric.device
        mat, vec = (lambda *n: self._mat(W, *n)), (lambda n: self._vec(W, n))
        self.embed, self.head, self.final_norm = mat("embed"), mat("head"), vec("final.norm")
        built: Dict[int, dict] = {}
        self.layers: List[dict] = []
        for i, l in enumerate(c.layers):
            j = c.owner(i)
            if j not in built:
                p, m = f"l{j}.", l.mixer
                cols = m.columns
                off = [0, cols[0], cols[0] + cols[1]]
                S = {"m": m, "norm1": vec(p + "norm1"), "in": mat(*[p + "mix." + n for n in "qkvg"]), "o": mat(p + "mix.o"), "off": off, "gate0": sum(cols[:3]),
                     "cols": sum(cols), "ff": l.ff}
                if l.ff:
                    S.update(norm2=vec(p + "norm2"), up=mat(p + "mlp.up"), down=mat(p + "mlp.down"))
                if m.recurrent:
                    ret = m.kind == "retention"
                    S["rec"] = DecayedMixer(heads=m.heads, dim=m.dim, vdim=m.vdim, decay=m.decay, offsets=off, device=dev, rot_dims=m.rot_dims,
                                            interleaved=False, act=None if ret else "silu", k_scale=m.dim ** -0.5 if ret else 1.0)
                    S["gain"] = None if ret else vec(p + "mix.norm")
                    S["groups"], S["gate_act"] = (m.heads, "silu") if ret else (1, "sigmoid")
                else:
                    S.update(q_norm=vec(p + "mix.q.norm"), k_norm=vec(p + "mix.k.norm"), sink=vec(p + "mix.sink"), gate_act="sigmoid")
                built[j] = S
            self.layers.append(dict(built[j]))        # shared tensors, own state

        # prompts: recurrences on the tensor cores in bf16 when every head fits a tile, f32 products otherwise
        self.tensor_recurrence = self.dtype == BF16 and all(max(l.mixer.dim, l.mixer.vdim) <= 128 for l in c.layers if l.mixer.recurrent)
        self.chunk = TILE if self.tensor_recurrence else CHUNK
        # the fused decode chain needs operand widths that are whole 16-byte chunks
        self.fused = self.dtype == BF16 and all(n % 8 == 0 for l in c.layers for n in (c.width, l.ff, l.mixer.heads * l.mixer.vdim))

    def _state_bytes(self) -> tuple:
        es = torch.empty((), dtype=self.dtype).element_size()
        att = [l.mixer for l in self.cfg.layers if not l.mixer.recurrent]
        rec = [l.mixer for l in self.cfg.layers if l.mixer.recurrent]
        return sum(m.kv_heads * (m.dim + m.vdim) for m in att) * es, sum(m.heads * m.dim * m.vdim for m in rec) * 4

    def _make_states(self) -> None:
        c, dev = self.cfg, self.fabric.device
        for L in self.layers:
            m = L["m"]
            if m.recurrent:
                L["state"] = L["rec"].state(self.num_slots, dev)
            else:
                L["k_cache"] = torch.zeros(self.num_pages, c.page_tokens, m.kv_heads, m.dim, dtype=self.dtype, device=dev)
                L["v_cache"] = torch.zeros(self.num_pages, c.page_tokens, m.kv_heads, m.vdim, dtype=self.dtype, device=dev)

    @classmethod
    def from_checkpoint(cls, path, fabric: Fabric, **kw) -> "FalinexDecoder":
        c, w = load_checkpoint(path)
        return cls(c, w, fabric, **kw)

    # -- layers ------------------------------------------------------------------------------------------------------------
    def _mix(self, B: _Rows, L: dict, m: int, pos, slot, plan: Optional[DevicePlan], norm: bool = True) -> None:
        """The mixer of one layer between its input projection (``B.proj``) and the operand of its output projection (``B.mixed``);
        ``plan``: of a packed step, None for decode rows. Without ``norm`` recurrent mixers leave their heads in ``B.o`` instead (the fused
        output projection norms and gates them)."""
        mx, st = L["m"], self.fabric.desc.status
        proj = B.proj[:m]
        hv = mx.heads * mx.vdim
        rope = B.rotary.get(mx.rot_dims, mx.rot_base)
        if mx.recurrent:
            o, rec, gate = B.o[:m, :hv], L["rec"], proj[:, L["gate0"]:L["gate0"] + hv]
            long = plan is not None and plan.table is not None
            alone = long and not plan.groups                       # every row belongs to a long run
            if long and self.tensor_recurrence:
                if alone and L["groups"] == mx.heads and L["gain"] is None:
                    rec.tiles(proj, L["state"], pos, plan.table, rope, B.scratch[3], gated=B.mixed[hv][:m], gate=gate, gate_act=L["gate_act"], eps=self.cfg.eps,
                              status_ptr=st)
                    return
                rec.tiles(proj, L["state"], pos, plan.table, rope, B.scratch[3], out=o, status_ptr=st)
            elif long:
                rec.chunks(proj, L["state"], pos, plan.table, rope, o, B.scratch)
            if not alone:
                rec.step(proj, L["state"], pos if plan is None else plan.step_positions, slot, rope, o)
            if norm:
                N.group_norm_gate(o, gate, L["gate_act"], self.cfg.eps, B.mixed[hv][:m], L["groups"], L["gain"])
            return
        q, out = B.q[mx.q_shape][:m], B.mixed[hv][:m]
        WA.qk_norm_rope_write(proj, L["off"], L["q_norm"], L["k_norm"], self.cfg.eps, heads=mx.heads, kv_heads=mx.kv_heads, dim=mx.dim, vdim=mx.vdim,
                              rot=mx.rot_dims, interleaved=True, rope=rope, positions=pos, slots=slot, page_table=self.page_table, q_out=q,
                              k_cache=L["k_cache"], v_cache=L["v_cache"], status_ptr=st)
        gate = proj[:, L["gate0"]:L["gate0"] + hv]
        how = dict(heads=mx.heads, window=mx.window, scale=mx.scale, sink=L["sink"], gate_act=L["gate_act"], status_ptr=st)
        caches = (L["k_cache"], L["v_cache"])
        tiled = plan is not None and bool(plan.runs) and mx.tiles and self.dtype == BF16
        if tiled:
            for r, n, sl, p0 in plan.runs:
                k, vt = B.ctx[mx.ctx_shape]
                WA.fa_window(q[r:r + n], *caches, self.page_table, slot=sl, pos0=p0, ctx_k=k, ctx_vt=vt, out=out[r:r + n], gate=gate[r:r + n], **how)
        groups = [(r, min(m, r + ATTN_ROWS)) for r in range(0, m, ATTN_ROWS)] if not tiled else plan.groups
        rest = plan.step_positions if tiled else pos
        if mx.splits and self.dtype == BF16:
            for lo, hi in groups:
                WA.gqa_window(q[lo:hi], *caches, rest[lo:hi], slot[lo:hi], self.page_table, splits=mx.splits, scratch=B.split_scratch, out=out[lo:hi],
                              gate=gate[lo:hi], **how)
        elif groups:
            WA.window_attn(q, *caches, rest, slot, self.page_table, out=out, gate=gate, **how)

    def _layers(self, B: _Rows, m: int, tok, pos, slot, plan: Optional[DevicePlan], final: bool, probe: Optional[list] = None) -> None:
        """All layers over ``m`` rows as separate row operators and matrix products; the residual ends in ``B.x``, and with ``final`` the
        normalised rows for the output matrix in ``B.xa``."""
        c, st, W = self.cfg, self.fabric.desc.status, self.cfg.width
        x, xa, y = B.x[:m, :W], B.xa[:m], B.y[:m, :W]
        N.embed_rows(tok, self.embed, x, xa, status_ptr=st)
        B.rotary.fill(pos)
        for i, L in enumerate(self.layers):
            mx = L["m"]
            hv = mx.heads * mx.vdim
            last = i + 1 == len(self.layers) and final
            N.linear(xa, L["in"], B.proj[:m, :L["cols"]], status_ptr=st)
            self._mix(B, L, m, pos, slot, plan)
            N.linear(B.mixed[hv][:m], L["o"], y, status_ptr=st)
            N.post_norm_add(y, L["norm1"], c.eps, x, xa, self.final_norm if last and not L["ff"] else None)
            if L["ff"]:
                N.linear(xa, L["up"], B.act[L["ff"]][:m, :L["ff"]], "gelu_tanh", status_ptr=st)
                N.linear(B.act[L["ff"]][:m], L["down"], y, status_ptr=st)
                N.post_norm_add(y, L["norm2"], c.eps, x, xa, self.final_norm if last else None)
            if probe is not None:
                probe.append(x.clone())

    def _layers_fused(self, B: _Rows, n: int, tok, pos, slot) -> None:
        """Decode rows: every norm, residual update, gate and activation inside the linear that follows or precedes it. Ends like
        :meth:`_layers` with ``final``."""
        c = self.cfg
        x, x2, xa, y = B.x[:n], B.x2[:n], B.xa[:n], B.y[:n]
        N.embed_rows(tok, self.embed, x, xa, status_ptr=self.fabric.desc.status)
        B.rotary.fill(pos)
        owed = None                            # gain of the sublayer output in y that the residual still lacks
        for L in self.layers:
            mx = L["m"]
            hv, proj = mx.heads * mx.vdim, B.proj[:n]
            if owed is None:
                N.gemv_act(xa, L["in"], proj)
            else:
                N.gemv_post_norm(y, owed, c.eps, x, x2, L["in"], proj)
                x, x2 = x2, x
            self._mix(B, L, n, pos, slot, None, norm=False)
            if mx.recurrent:
                N.gemv_group_norm(B.o[:n, :hv], proj[:, L["gate0"]:], L["gate_act"], c.eps, L["o"], y, L["groups"], L["gain"])
            else:
                N.gemv_act(B.mixed[hv][:n], L["o"], y)
            owed = L["norm1"]
            if L["ff"]:
                act = B.act[L["ff"]][:n]
                N.gemv_post_norm(y, owed, c.eps, x, x2, L["up"], act, "gelu_tanh")
                x, x2 = x2, x
                N.gemv_act(act, L["down"], y)
                owed = L["norm2"]
        N.post_norm_add(y, owed, c.eps, x, xa, self.final_norm)


class FalinexRows(StreamRows):
    """Packed-step executor: see :class:`StreamRows`."""
