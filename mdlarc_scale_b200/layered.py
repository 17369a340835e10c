"""Layered models on the engine: the network as data, its session (cache, recurrent state, slots) and the
packing of mixed batches of prompt portions and single tokens."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

import numpy as np
import torch

from . import _lib
from .engine import EngineBase, Session, _ptr, _stream_ptr

QBLOCK = 256    # query rows of one tile pair of the prefill attention


@dataclass(frozen=True)
class LayerSpec:
    """One layer: a token mixer and an optional feed-forward (``arcb_layer_desc``)."""
    mixer: str                  # "attention" | "mlstm" | "latent"
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    kv_from: int = -1
    qkv_bias: bool = False
    qk_norm: bool = False
    sink: bool = False
    out_gate: bool = False
    scale: float = 1.0
    q_temp_coef: float = 0.0
    q_temp_every: int = 0
    gate_cap: float = 1.0
    mlp: str | None = None      # "relu2" | "glu" | "moe" | None
    d_ff: int = 0               # hidden size (of one expert)
    window: int = 0             # positions an attention layer sees, its own included; 0: all before it
    q_rank: int = 0             # latent attention: query latent, cached latent, rotated key part
    kv_rank: int = 0
    rot_dim: int = 0
    rot_dims: int = 0           # rotated dimensions of that part
    rot_base: float = 10000.0
    glu: str = "silu"           # "silu" | "clamped"
    glu_limit: float = 0.0
    experts: int = 0
    top: int = 0
    shared_ff: int = 0
    shared_limit: float = 0.0


@dataclass(frozen=True)
class ModelSpec:
    width: int
    vocab: int
    layers: list[LayerSpec]
    norm: str = "layer"         # "layer" | "rms"
    norm_eps: float = 1e-6
    residual_alpha: float = 1.0
    logit_scale: float = 1.0
    norm_place: str = "post"    # "post": after the sums | "sandwich": before and after every sublayer
    loop: tuple[int, int, int] = (0, 0, 1)     # layers start .. stop - 1 run `times` times

    @property
    def n_runs(self) -> int:
        start, stop, times = self.loop
        return len(self.layers) + (times - 1) * (stop - start)


class LayeredEngine(EngineBase):
    """Packed weights of a layered model.  ``tensors`` maps (kind, layer) to fp32-convertible tensors in
    [out, in] order, or to the list of them that a stacked kind wants; the kinds are those of
    ``_lib.LAYERED_KINDS``."""

    end_token = -1

    def __init__(self, spec: ModelSpec, tensors: dict[tuple[str, int], torch.Tensor], device="cuda:0",
                 act_format: str = "f16", gemm_path: str = "auto", attn_path: str = "auto", mlstm_path: str = "auto",
                 fused_proj: bool = True):
        super().__init__(device)
        self.spec = spec
        self.vocab_size = spec.vocab
        self.n_layers = len(spec.layers)
        self.act_format = {"f16": _lib.ACT_F16, "bf16": _lib.ACT_BF16, "f32": _lib.ACT_F32}[act_format]
        md = _lib.ModelDesc(
            width=spec.width, vocab=spec.vocab, n_layers=self.n_layers, norm_place=_lib.PLACES[spec.norm_place],
            loop_start=spec.loop[0], loop_stop=spec.loop[1], loop_times=spec.loop[2], norm=_lib.NORMS[spec.norm],
            act_format=self.act_format, gemm_path={"auto": _lib.GEMM_AUTO, "simt": _lib.GEMM_SIMT}[gemm_path],
            attn_path={"auto": _lib.ATTN_AUTO, "stream": _lib.ATTN_STREAM}[attn_path],
            mlstm_path={"auto": _lib.MLSTM_AUTO, "step": _lib.MLSTM_STEP}[mlstm_path], fused_proj=int(bool(fused_proj)),
            norm_eps=spec.norm_eps, residual_alpha=spec.residual_alpha, logit_scale=spec.logit_scale)
        ld = (_lib.LayerDesc * self.n_layers)(*[
            _lib.LayerDesc(
                mixer=_lib.MIXERS[s.mixer], heads=s.heads, kv_heads=s.kv_heads, dim=s.dim, vdim=s.vdim, kv_from=s.kv_from,
                qkv_bias=int(s.qkv_bias), qk_norm=int(s.qk_norm), sink=int(s.sink), out_gate=int(s.out_gate),
                scale=s.scale, q_temp_coef=s.q_temp_coef, q_temp_every=s.q_temp_every, gate_cap=s.gate_cap,
                mlp=_lib.MLPS[s.mlp], d_ff=s.d_ff, window=s.window, q_rank=s.q_rank, kv_rank=s.kv_rank, rot_dim=s.rot_dim,
                rot_dims=s.rot_dims, rot_base=s.rot_base, glu=_lib.GLUS[s.glu], glu_limit=s.glu_limit, experts=s.experts,
                top=s.top, shared_ff=s.shared_ff, shared_limit=s.shared_limit) for s in spec.layers])
        with torch.cuda.device(self.device):
            _lib.check(self.lib.arcb_engine_create_layered(C.byref(md), ld, C.byref(self._handle)))
            for (kind, layer), t in tensors.items():
                if isinstance(t, list):
                    t = torch.stack([x.to(self.device) for x in t])
                self._load_id(_lib.LAYERED_KIND[kind], layer, t)
            torch.cuda.synchronize(self.device)


@dataclass
class Segment:
    """The next tokens of the sequence in ``slot``; ``want``: places among them whose logits are asked for."""
    slot: int
    tokens: list[int] | np.ndarray
    want: list[int] = field(default_factory=list)
    arm: bool = False           # pick the first generated token from the last row and start decoding


@dataclass
class PackedSegments:
    """One prefill call's integer arrays, laid out in one host buffer that reaches the device in one copy."""
    buf: torch.Tensor
    at: dict[str, tuple[int, int]]
    n_tokens: int
    n_segs: int
    n_want: int
    n_first: int
    n_qblocks: int
    group_qblock: np.ndarray | None = None     # expansion groups: first query block and first tile of each
    group_tile: np.ndarray | None = None

    @property
    def n_groups(self) -> int:
        return 0 if self.group_tile is None else len(self.group_tile) - 1

    def ptr(self, dev: torch.Tensor, name: str) -> int | None:
        lo, n = self.at[name]
        return dev.data_ptr() + 4 * lo if n else None


def plan_expansion(blocks: list[tuple[int, int, int, int]], window: int, rows: int):
    """Groups query blocks so that the keys and values each group needs, expanded from cached latents, fit a scratch
    of ``rows`` rows.  ``blocks``: (segment, position of the first row, number of rows, packed row) in segment order.
    Within a group a segment's keys are consecutive scratch rows that start on a tile of 128.  Returns one
    (blocks, tiles, kv0) per group: block indices, (segment, position) of every tile's first row, and the scratch row
    that position 0 of each block's sequence would have."""
    groups, cur = [], None
    for i, (seg, p0, n, _) in enumerate(blocks):
        lo, hi = max(0, p0 - window + 1), p0 + n
        while True:
            if cur is None:
                cur = {"blocks": [], "runs": [], "tiles": 0}
            run = cur["runs"][-1] if cur["runs"] and cur["runs"][-1][0] == seg else None
            first, base = (run[1], run[2]) if run else (lo, cur["tiles"])
            tiles = base + -(-(hi - first) // 128)
            if tiles * 128 <= rows:
                break
            if not cur["blocks"]:
                raise ValueError("a query block and its window exceed the expansion scratch")
            groups.append(cur)
            cur = None
        if run is None:
            cur["runs"].append([seg, lo, base])
        cur["blocks"].append((i, base * 128 - first))
        cur["tiles"] = tiles
    if cur is not None:
        groups.append(cur)
    out = []
    for g in groups:
        ends = [r[2] for r in g["runs"][1:]] + [g["tiles"]]
        tiles = [(seg, first + 128 * t) for (seg, first, base), end in zip(g["runs"], ends) for t in range(end - base)]
        out.append(([b for b, _ in g["blocks"]], tiles, [k for _, k in g["blocks"]]))
    return out


def pack_segments(segments: list[Segment], pos0: list[int], expand: tuple[int, int, int] | None = None) -> PackedSegments:
    """Packs portions of several sequences back to back.  Row arrays: token, cache row, position (= cache
    slot) and visible keys; segment arrays; the rows asked for; and the query blocks of the prefill
    attention, most expensive first (their CTAs are dispatched in that order).  ``expand``: scratch rows, widest
    window and cache row pitch of a model with latent attention, whose blocks are grouped (plan_expansion)."""
    rows = np.array([len(s.tokens) for s in segments], np.int64)
    row0 = np.concatenate([[0], np.cumsum(rows)[:-1]]).astype(np.int64)
    slot = np.array([s.slot for s in segments], np.int64)
    p0 = np.array(pos0, np.int64)
    seg_of = np.repeat(np.arange(len(segments)), rows)
    pos = np.arange(int(rows.sum())) - row0[seg_of] + p0[seg_of]
    want = [int(row0[i]) + int(w) for i, s in enumerate(segments) for w in s.want]
    for i, s in enumerate(segments):
        if any(w < 0 or w >= rows[i] for w in s.want):
            raise ValueError("a wanted place lies outside its portion")
    arm = [i for i, s in enumerate(segments) if s.arm]
    blocks = [(i, int(p0[i]) + r, int(min(QBLOCK, rows[i] - r)), int(row0[i]) + r)
              for i in range(len(segments)) for r in range(0, int(rows[i]), QBLOCK)]
    if expand is None:
        groups = [(list(range(len(blocks))), [], [0] * len(blocks))]
    else:
        groups = plan_expansion(blocks, expand[1], expand[0])
    order, kv0, tile_src, group_qblock, group_tile = [], [], [], [0], [0]
    for members, tiles, starts in groups:
        by_cost = sorted(range(len(members)), key=lambda k: -(blocks[members[k]][1] + blocks[members[k]][2]))
        order += [members[k] for k in by_cost]
        kv0 += [starts[k] for k in by_cost]
        tile_src += [int(slot[seg]) * (expand[2] if expand else 0) + p for seg, p in tiles]
        group_qblock.append(len(order))
        group_tile.append(len(tile_src))
    blocks = [(blocks[i][3], blocks[i][2]) for i in order]
    arrays = {
        "token": np.concatenate([np.asarray(s.tokens, np.int64) for s in segments]),
        "seq": slot[seg_of], "pos": pos, "count": pos + 1,
        "seg_row0": row0, "seg_rows": rows, "seg_seq": slot, "seg_pos0": p0,
        "want": want, "first_row": [int(row0[i] + rows[i] - 1) for i in arm], "first_seq": slot[arm] if arm else [],
        "first_len": [int(p0[i] + rows[i]) for i in arm],
        "qb_row0": [b[0] for b in blocks], "qb_rows": [b[1] for b in blocks],
        "qb_kv0": kv0, "tile_src": tile_src + tile_src[-1:],      # one spare: tiles are read in pairs
    }
    at, parts, off = {}, [], 0
    for name, v in arrays.items():
        v = np.asarray(v, np.int32)
        at[name] = (off, len(v))
        pad = -len(v) % 4                     # every array starts on a 16-byte boundary
        parts.append(v)
        if pad:
            parts.append(np.zeros(pad, np.int32))
        off += len(v) + pad
    packed = PackedSegments(torch.from_numpy(np.concatenate(parts)), at, int(rows.sum()), len(segments), len(want),
                            len(arm), len(blocks))
    if expand is not None:
        packed.group_qblock, packed.group_tile = np.array(group_qblock, np.int32), np.array(group_tile, np.int32)
    return packed


class LayeredSession(Session):
    """Session of a layered model: slots of a cache that holds keys, values and recurrent states, all
    continued from call to call.  ``lens[slot]`` is the number of positions the slot holds."""

    def __init__(self, *args, **kw):
        super().__init__(*args, **kw)
        self.lens = [0] * self.n_seqs
        self._free = list(range(self.n_seqs - 1, -1, -1))
        rows, window = C.c_int32(), C.c_int32()
        _lib.check(self.eng.lib.arcb_session_expand_rows(self._handle, C.byref(rows), C.byref(window)))
        self._expand = (rows.value, window.value, self.t_max) if rows.value else None
        if self.step_logits is not None and self.palette_mask is not None:
            raise ValueError("grid constraints do not apply to layered models")

    # -- slots ----------------------------------------------------------------
    def acquire(self) -> int:
        if not self._free:
            raise RuntimeError("no free slot in the session")
        slot = self._free.pop()
        self.lens[slot] = 0
        return slot

    def release(self, slot: int) -> None:
        if slot in self._free:
            raise ValueError(f"slot {slot} is already free")
        self.lens[slot] = 0
        self._free.append(slot)

    @property
    def free_slots(self) -> int:
        return len(self._free)

    # -- compute --------------------------------------------------------------
    def _check(self, slot: int, n: int) -> None:
        if slot < 0 or slot >= self.n_seqs:
            raise ValueError(f"slot {slot} outside the session")
        if n <= 0:
            raise ValueError("a portion must have at least one token")
        if self.lens[slot] + n > self.t_max:
            raise ValueError(f"slot {slot} would hold {self.lens[slot] + n} positions, the session has {self.t_max}")

    def prefill_segments(self, segments: list[Segment], logits_all: bool = False, residuals: bool = False):
        """One forward over portions of one or more sequences.  Returns (logits of the wanted rows in
        segment order or of all rows, first-token logits of the armed segments, residual stream after every
        layer run), each None when not asked for."""
        slots = [s.slot for s in segments]
        if len(set(slots)) != len(slots):
            raise ValueError("a sequence may appear once in a call")
        for s in segments:
            self._check(s.slot, len(s.tokens))
        p = pack_segments(segments, [self.lens[s.slot] for s in segments], self._expand)
        if p.n_tokens > self.max_prefill_tokens:
            raise ValueError("the call has more tokens than the session's prefill capacity")
        dev, V = self.eng.device, self.eng.vocab_size
        buf = p.buf.to(dev, non_blocking=True)
        f32 = dict(dtype=torch.float32, device=dev)
        everything = torch.empty((p.n_tokens, V), **f32) if logits_all else None
        wanted = torch.empty((p.n_want, V), **f32) if p.n_want else None
        first = torch.empty((p.n_first, V), **f32) if p.n_first else None
        res = torch.empty((self.eng.spec.n_runs, p.n_tokens, self.eng.spec.width), **f32) if residuals else None
        a = _lib.PrefillArgs(
            n_tokens=p.n_tokens, d_token_ids=p.ptr(buf, "token"), d_seq=p.ptr(buf, "seq"), d_kv_slot=p.ptr(buf, "pos"),
            d_kv_count=p.ptr(buf, "count"), n_qblocks=p.n_qblocks, d_qblock_row0=p.ptr(buf, "qb_row0"),
            d_qblock_rows=p.ptr(buf, "qb_rows"), d_logits_all=_ptr(everything), n_first=p.n_first,
            d_first_row=p.ptr(buf, "first_row"), d_first_seq=p.ptr(buf, "first_seq"), d_prompt_len=p.ptr(buf, "first_len"),
            d_first_logits=_ptr(first), n_segs=p.n_segs, d_seg_row0=p.ptr(buf, "seg_row0"), d_seg_rows=p.ptr(buf, "seg_rows"),
            d_seg_seq=p.ptr(buf, "seg_seq"), d_seg_pos0=p.ptr(buf, "seg_pos0"), n_logit_rows=p.n_want,
            d_logit_row=p.ptr(buf, "want"), d_logits=_ptr(wanted), d_residuals=_ptr(res))
        if p.n_groups:
            a.d_qblock_kv0, a.d_tile_src, a.n_groups = p.ptr(buf, "qb_kv0"), p.ptr(buf, "tile_src"), p.n_groups
            a.h_group_qblock, a.h_group_tile = p.group_qblock.ctypes.data, p.group_tile.ctypes.data
        with torch.cuda.device(dev):
            _lib.check(self.eng.lib.arcb_prefill(self._handle, C.byref(a), _stream_ptr(dev)))
        for s in segments:
            self.lens[s.slot] += len(s.tokens)
        return (everything if logits_all else wanted), first, res

    def feed(self, slots: list[int], tokens: list[int]) -> torch.Tensor:
        """One decode step (the captured graph) with the given tokens for the given slots; all other slots
        hold still.  Returns the step's logits [len(slots), vocab]."""
        if len(set(slots)) != len(slots):
            raise ValueError("a sequence may appear once in a step")
        for s in slots:
            self._check(s, 1)
        dev = self.eng.device
        buf = torch.tensor([*slots, *tokens], dtype=torch.int32).to(dev, non_blocking=True)
        with torch.cuda.device(dev):
            _lib.check(self.eng.lib.arcb_session_feed(self._handle, len(slots), buf.data_ptr(),
                                                      buf.data_ptr() + 4 * len(slots), _stream_ptr(dev)))
        self.decode(1)
        for s in slots:
            self.lens[s] += 1
        return self.last_logits()[buf[:len(slots)].long()]

    def last_logits(self) -> torch.Tensor:
        """View of the last decode step's logits, [n_seqs, vocab]; the next call overwrites it."""
        ptr, pitch = C.c_void_p(), C.c_int32()
        _lib.check(self.eng.lib.arcb_session_step_logits(self._handle, C.byref(ptr), C.byref(pitch)))
        off = ptr.value - self.workspace.data_ptr()
        rows = self.workspace[off:off + self.n_seqs * pitch.value * 4].view(torch.float32)
        return rows.view(self.n_seqs, pitch.value)[:, :self.eng.vocab_size]

    def step(self, segments: list[Segment]) -> list[torch.Tensor | None]:
        """Advances every named sequence by its portion: single tokens of started sequences through the decode
        step, anything else through prefill.  Per segment the logits of its wanted places (or None)."""
        if all(len(s.tokens) == 1 and self.lens[s.slot] > 0 for s in segments):
            rows = self.feed([s.slot for s in segments], [int(s.tokens[0]) for s in segments])
            return [rows[i:i + 1].clone() if s.want else None for i, s in enumerate(segments)]
        out: list[list[torch.Tensor]] = [[] for _ in segments]
        done = [0] * len(segments)
        while True:
            call, owner, room = [], [], self.max_prefill_tokens
            for i, s in enumerate(segments):
                n = min(len(s.tokens) - done[i], room)
                if n > 0:
                    want = [w - done[i] for w in s.want if done[i] <= w < done[i] + n]
                    call.append(Segment(s.slot, s.tokens[done[i]:done[i] + n], want, s.arm and done[i] + n == len(s.tokens)))
                    owner.append(i)
                    done[i] += n
                    room -= n
            if not call:
                break
            logits, _, _ = self.prefill_segments(call)
            at = 0
            for i, c in zip(owner, call):
                if c.want:
                    out[i].append(logits[at:at + len(c.want)])
                    at += len(c.want)
        return [torch.cat(o) if o else None for o in out]

    def finished(self) -> np.ndarray:
        """Flags of the slots that have emitted the end token or used up ``max_new`` (synchronises)."""
        flags = np.zeros(self.n_seqs, np.int32)
        dev = self.eng.device
        with torch.cuda.device(dev):
            _lib.check(self.eng.lib.arcb_session_finished(self._handle, flags.ctypes.data, _stream_ptr(dev)))
        return flags


LayeredEngine.session_class = LayeredSession
