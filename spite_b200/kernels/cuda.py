"""`CudaKernels`: the product kernel set.  Hand-written CUDA for sm_100a under
`spite_b200/csrc`, compiled in-tree and called through ctypes on the current
torch stream.  There is no other implementation in the package: without a CUDA
device or without the compiled libraries every call raises.
"""
from __future__ import annotations

import collections
import ctypes as C
import math
import os

import torch

from . import build
from .api import KernelError, KernelSet, KernelTimeout, Routing

_DT = {torch.float32: 0, torch.bfloat16: 1}
_STATUS = {-1: "malformed argument", -2: "size not supported by this kernel", -3: "launch failed"}

EPI_STORE, EPI_STORE_F32, EPI_ADD_F32, EPI_SWIGLU = 0, 1, 2, 3
_WINDOW = {"full": 0, "chunk": 1, "sliding": 2}
_ACTIVATION = {None: 0, "relu2": 1, "gelu_tanh": 2, "xielu": 3, "tanh": 4}


class GemmParams(C.Structure):
    _fields_ = [("A", C.c_void_p), ("W", C.c_void_p), ("C", C.c_void_p),
                ("a_rows", C.c_void_p), ("c_rows", C.c_void_p), ("group_offsets", C.c_void_p),
                ("row_scale", C.c_void_p),
                ("lda", C.c_longlong), ("ldc", C.c_longlong), ("w_group_stride", C.c_longlong),
                ("n_groups", C.c_int), ("M", C.c_int), ("N", C.c_int), ("K", C.c_int),
                ("epilogue", C.c_int), ("scale_by_a_row", C.c_int), ("activation", C.c_int),
                ("bias", C.c_void_p), ("act_pos", C.c_float), ("act_neg", C.c_float)]


class StepTokens(C.Structure):
    _fields_ = [("positions", C.c_void_p), ("seg_of_token", C.c_void_p), ("block_table", C.c_void_p),
                ("table_width", C.c_int), ("n_tokens", C.c_int)]


class PagedCache(C.Structure):
    _fields_ = [("kv", C.c_void_p), ("v_offset", C.c_longlong), ("n_pages", C.c_int),
                ("page_size", C.c_int), ("num_kv_heads", C.c_int), ("head_dim", C.c_int), ("key_scale", C.c_void_p)]


class QkPrepareParams(C.Structure):
    _fields_ = [("qkv", C.c_void_p), ("q_out", C.c_void_p), ("inv_freq", C.c_void_p),
                ("q_gain", C.c_void_p), ("k_gain", C.c_void_p),
                ("qk_norm_eps", C.c_float), ("norm_before_rotation", C.c_int), ("pairing", C.c_int),
                ("rotary_dim", C.c_int), ("temperature_floor", C.c_int),
                ("temperature_scale", C.c_float), ("num_heads", C.c_int), ("write_cache", C.c_int),
                ("qkv_stride", C.c_longlong), ("rot_amplitude", C.c_float),
                ("v_other", C.c_void_p), ("v_other_stride", C.c_longlong), ("v_other_head", C.c_int),
                ("v_mix_dim", C.c_int), ("v_mix", C.c_float), ("gates_out", C.c_void_p),
                ("bias", C.c_void_p), ("q_only", C.c_int), ("norm_dim", C.c_int),
                ("v_inv_freq", C.c_void_p), ("v_rotary_dim", C.c_int), ("v_pairing", C.c_int),
                ("inv_freq_low", C.c_void_p), ("v_inv_freq_low", C.c_void_p), ("values_are_keys", C.c_int)]


class AttentionParams(C.Structure):
    _fields_ = [("q", C.c_void_p), ("out", C.c_void_p), ("num_heads", C.c_int),
                ("window_kind", C.c_int), ("window_size", C.c_int), ("softmax_scale", C.c_float),
                ("has_sink", C.c_int), ("sink_logit", C.c_float),
                ("head_sinks", C.c_void_p), ("head_slopes", C.c_void_p), ("head_gates", C.c_void_p),
                ("out_by_head_tokens", C.c_int), ("score_softcap", C.c_float),
                ("distance_bias", C.c_void_p), ("distance_runs", C.c_void_p), ("distance_len", C.c_int)]


class LatentPrepareParams(C.Structure):
    _fields_ = [("down", C.c_void_p), ("down_stride", C.c_longlong), ("cq_out", C.c_void_p),
                ("q_gain", C.c_void_p), ("kv_gain", C.c_void_p), ("inv_freq", C.c_void_p),
                ("rot_amplitude", C.c_float), ("eps", C.c_float),
                ("q_rank", C.c_int), ("kv_rank", C.c_int), ("rot_dim", C.c_int), ("num_gates", C.c_int),
                ("gates_out", C.c_void_p), ("write_cache", C.c_int), ("pairing", C.c_int)]


class LatentQueryParams(C.Structure):
    _fields_ = [("q", C.c_void_p), ("q_out", C.c_void_p), ("inv_freq", C.c_void_p), ("rot_amplitude", C.c_float),
                ("num_heads", C.c_int), ("head_dim", C.c_int), ("rot_dim", C.c_int), ("kv_rank", C.c_int),
                ("row", C.c_int), ("positions", C.c_void_p), ("n_tokens", C.c_int),
                ("rows_out", C.c_void_p), ("offsets_out", C.c_void_p), ("q_sorted_out", C.c_void_p), ("pairing", C.c_int)]


class ShortConvParams(C.Structure):
    _fields_ = [("x", C.c_void_p), ("x_stride", C.c_longlong), ("w", C.c_void_p), ("out", C.c_void_p),
                ("out_stride", C.c_longlong), ("state", C.c_void_p), ("slot_stride", C.c_longlong),
                ("cu_seqlens", C.c_void_p), ("slots", C.c_void_p), ("n_segments", C.c_int), ("channels", C.c_int),
                ("taps", C.c_int), ("copy_columns", C.c_int), ("activation", C.c_int), ("max_seg_len", C.c_int),
                ("bias", C.c_void_p)]


class TokenShiftParams(C.Structure):
    _fields_ = [("x", C.c_void_p), ("mu", C.c_void_p), ("out", C.c_void_p), ("state", C.c_void_p),
                ("slot_stride", C.c_longlong), ("seg_of_token", C.c_void_p), ("cu_seqlens", C.c_void_p),
                ("slots", C.c_void_p), ("offsets_out", C.c_void_p), ("n_tokens", C.c_int), ("d", C.c_int),
                ("n_mixes", C.c_int)]


class StreamsParams(C.Structure):
    _fields_ = [("x", C.c_void_p), ("y", C.c_void_p), ("bias", C.c_void_p), ("scale", C.c_void_p), ("mix", C.c_void_p),
                ("w_out", C.c_void_p), ("w_in", C.c_void_p), ("gain", C.c_void_p), ("next_out", C.c_void_p),
                ("rows", C.c_void_p), ("n_rows", C.c_int), ("d", C.c_int), ("streams", C.c_int), ("write_back", C.c_int),
                ("eps", C.c_float)]


class ScanParams(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p),
                ("q_stride", C.c_longlong), ("k_stride", C.c_longlong), ("v_stride", C.c_longlong),
                ("w", C.c_void_p), ("w_stride", C.c_longlong), ("scalars", C.c_void_p), ("skip", C.c_void_p),
                ("out", C.c_void_p), ("out_stride", C.c_longlong), ("state", C.c_void_p), ("slot_stride", C.c_longlong),
                ("cu_seqlens", C.c_void_p), ("slots", C.c_void_p), ("n_segments", C.c_int), ("n_tokens", C.c_int),
                ("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int), ("out_scale", C.c_float)]


class DeltaParams(C.Structure):
    _fields_ = [("x", C.c_void_p), ("stride", C.c_longlong),
                ("q_col", C.c_int), ("k_col", C.c_int), ("v_col", C.c_int), ("b_col", C.c_int), ("a_col", C.c_int),
                ("a_log", C.c_void_p), ("dt_bias", C.c_void_p), ("out", C.c_void_p), ("state", C.c_void_p),
                ("slot_stride", C.c_longlong), ("cu_seqlens", C.c_void_p), ("slots", C.c_void_p),
                ("n_segments", C.c_int), ("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int),
                ("q_scale", C.c_float), ("unit_eps", C.c_float), ("gates", C.c_void_p), ("n_tokens", C.c_int)]


class MlstmParams(C.Structure):
    _fields_ = [("proj", C.c_void_p), ("stride", C.c_longlong),
                ("q_col", C.c_int), ("k_col", C.c_int), ("v_col", C.c_int), ("i_col", C.c_int), ("f_col", C.c_int),
                ("i_bias", C.c_void_p), ("f_bias", C.c_void_p), ("out", C.c_void_p), ("state", C.c_void_p),
                ("head_stride", C.c_longlong), ("cu_seqlens", C.c_void_p), ("slots", C.c_void_p),
                ("n_segments", C.c_int), ("heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int),
                ("gate_cap", C.c_float), ("q_scale", C.c_float), ("chunked", C.c_int)]


class AttnMmaExtra(C.Structure):
    _fields_ = [("cu_seqlens", C.c_void_p), ("o_part", C.c_void_p), ("ml_part", C.c_void_p),
                ("n_segments", C.c_int), ("tokens_per_block", C.c_int), ("n_splits", C.c_int),
                ("seg_min_tokens", C.c_int), ("seg_max_tokens", C.c_int)]


class AttnDecodeExtra(C.Structure):
    _fields_ = [("cu_seqlens", C.c_void_p), ("partial", C.c_void_p), ("tickets", C.c_void_p),
                ("n_segments", C.c_int), ("tokens_per_block", C.c_int), ("n_splits", C.c_int),
                ("seg_min_tokens", C.c_int), ("seg_max_tokens", C.c_int), ("cache_settled", C.c_int)]


class SampleParams(C.Structure):
    _fields_ = [("logits", C.c_void_p), ("work", C.c_void_p), ("temperature", C.c_void_p),
                ("top_k", C.c_void_p), ("top_p", C.c_void_p), ("min_p", C.c_void_p),
                ("repetition_penalty", C.c_void_p), ("context", C.c_void_p),
                ("context_offsets", C.c_void_p), ("rng_state", C.c_void_p),
                ("out_tokens", C.c_void_p), ("vocab", C.c_int)]


# Libraries whose kernels wait on mbarriers with a limit.  A kernel that gives up records a code in its
# library's word of one small buffer in pinned host memory, which the device writes directly: the host
# reads it after any point at which it has waited for a step's results, without another copy or wait.
_WAITING_LIBRARIES = ("gemm_tc", "gemm_tc_pair", "gemm_stream", "attention_tc", "attention_decode", "gemm_tc_experts")
_error_words = None          # pinned int32 [len(_WAITING_LIBRARIES)], one per process
_configured: set = set()


def _error_buffer():
    global _error_words
    if _error_words is None:
        _error_words = torch.zeros(len(_WAITING_LIBRARIES), dtype=torch.int32).pin_memory()
    return _error_words


def _ptr(t):
    return None if t is None else t.data_ptr()


def _check(status, what):
    if status != 0:
        raise KernelError(f"{what}: {_STATUS.get(status, f'status {status}')}")


def stream_cut(M: int, N: int, K: int, groups: int, swiglu: bool, slots: int, smem: int, nt: int, *,
               item_cost: float = 2.0, split_item_cost: float = 6.0, split_cost: float = 1.5, slice_cost: float = 1.0,
               max_slices: int = 8, slices_min_rows: int = 4, cluster_max_splits: int = 0, cluster_cost: float = 0.0):
    """(k slices inside a block, k splits across blocks) of the weight-streaming kernel for a product of M rows,
    N output columns (per group) and depth K on `slots` resident blocks of `smem` bytes, `nt` token columns.

    A product of few tiles of 128 rows (a dense projection at a few tokens: 40 to 128 tiles for 296 to 444
    resident blocks) would leave most multiprocessors without work, and the ones that have some are then
    bound by what a single one can pull; so the items are made smaller until they fill the resident blocks
    about once: lower tiles with the k blocks of a stage side by side (the sums meet in shared memory), or k
    splits across blocks (partial sums through global memory, a ticket, a second pass over as many partial
    tiles as there are splits).  The cost of a choice is its rounds of items times (stages an item + what an
    item costs besides, in stages of 16 KiB: `item_cost` for any item, `split_item_cost` + `split_cost` a split
    if its sums cross blocks through global memory, `cluster_cost` if the splits, no more than
    `cluster_max_splits`, can be one thread-block cluster with all clusters resident at once, `slice_cost` if
    its slices meet in shared memory); at least four stages stay together.

    Measured on B200, us, (slices, splits) forced, each product alone.  Eight tokens (444 blocks): qkv 7168 x
    5120: (1, 5) 19.6, (2, 1) 20.9, (4, 1) 17.3, (8, 1) 21.3, (2, 2) 18.9; output projection 5120 x 5120: (1, 7)
    16.5, (4, 1) 14.2, (8, 1) 13.0, (4, 2) 13.1; shared down 5120 x 8192: (1, 7) 21.6, (4, 1) 20.8, (8, 1) 18.6;
    seven experts' gate/up: (1, 1) 220, (1, 2) 199.5, (2, 1) 197.4, (4, 1) 195.5; their down product: (1, 1)
    117.6, (2, 1) 113.5, (4, 1) 107.3, (8, 1) 113.4.  One token (296 blocks with rings twice as deep): slices
    bring nothing, qkv (1, 5) 17.5, (2, 2) 17.0, (4, 1) 19.5; output projection (1, 7) 13.9, (2, 2) 14.1, (4, 1)
    17.1.  In the decode step (ms at 4 / 6 / 8 / 12 / 16 tokens): no slices 4.64 / 5.64 / 6.63 / 8.38 / 9.67;
    slices everywhere 4.89 / 5.85 / 6.51 / 8.68 / 9.45; for one-group products only 4.73 / 5.62 / 6.52 / 8.41 /
    9.53; for the experts' products only 4.76 / 5.83 / 6.63 / 8.68 / 9.60.  The experts' products are faster
    alone with slices and slower in the step: with tiles of 128 rows some blocks end early and the next
    kernel's blocks start under the rest.  So the caller allows slices for one-group products from
    `slices_min_rows` rows on (the kernel set's defaults: six), and tiles of 128 rows otherwise."""
    best, best_cost = (1, 1), None
    for slices in (1, 2, 4, 8):
        if K % (64 * slices) or (swiglu and slices == 8):
            continue
        if slices > 1 and (M < slices_min_rows or slices > max_slices):
            continue
        stage_bytes = 16384 + max(1024, slices * nt * 128)
        if slices > 1 and (smem - 5504 - (8 - 8 // slices) * 64 * nt) // stage_bytes < 2:
            continue                                          # a ring of one stage
        rows = 128 // slices
        tiles = -(-N // (rows // 2 if swiglu else rows)) * groups
        stages = K // (64 * slices)
        for s in range(1, max(1, min(32, stages // 4)) + 1):
            rounds = -(-tiles * s // slots)
            fixed = item_cost + (slice_cost if slices > 1 else 0.0)
            if s > 1 and slices == 1 and s <= cluster_max_splits and tiles * s <= slots:
                fixed += cluster_cost                         # the splits as one cluster: their sums meet in shared memory
            elif s > 1:
                fixed += split_item_cost + split_cost * s
            cost = rounds * (-(-stages // s) + fixed)
            if best_cost is None or cost < best_cost:
                best, best_cost = (slices, s), cost
            if tiles * s >= 4 * slots:
                break
    return best


class CudaKernels(KernelSet):
    def __init__(self, dtype: torch.dtype, device="cuda:0"):
        if dtype not in _DT:
            raise KernelError(f"no kernel set for {dtype}; use torch.bfloat16 or torch.float32")
        if not torch.cuda.is_available():
            raise KernelError("spite_b200 needs a CUDA device (sm_100a); there is no CPU path")
        self.dtype = dtype
        self.device = torch.device(device)
        self._dt = _DT[dtype]
        self._libs = {}
        self.launches = 0          # kernels launched so far (for measurement reports)
        self.attention_scratch_bytes = 0   # partial results of the last split-key attention call
        self.launches_by_library = collections.Counter()   # the same, by kernel library
        self.sm_count = torch.cuda.get_device_properties(self.device).multi_processor_count
        # Which kernel takes which shape.  The numbers are measured choices (what was measured stands beside
        # each); they are plain attributes, so a measurement script can set another value on the object.
        # One switch is read from the environment, for finding a fault: SPITE_NO_TCGEN05=1 keeps every
        # tcgen05 kernel (products and attention) out, and shapes fall to the mma.sync and CUDA-core kernels.
        no_tc = os.environ.get("SPITE_NO_TCGEN05", "") not in ("", "0")
        self.use_tcgen05 = not no_tc
        self.use_tcgen05_attention = not no_tc
        self.attention_tc_min_tokens = 0       # fewest tokens of a request in a step that go to the tcgen05 attention (0: one full tile of rows)
        # most key splits of decode attention: beyond about twenty the merge by the last block costs more than the
        # extra blocks bring (one request at 8,192 keys: 22 us with 37 splits, 17.6 us with 18)
        self.attention_max_splits = 24
        self.attention_narrow_rows = 8         # decoded tokens of up to so many heads a kv head take its form of eight rows (0: never)
        self.use_decode_attention = True       # the TMA-fed decode kernel (head sizes 64 and 128, pages of a multiple of 64 keys)
        # row counts up to which the weight-streaming kernel is preferred over the tcgen05 one
        self.skinny_max_rows = 16
        self.skinny_blocks = 2 * self.sm_count
        # one-group products of at least this many rows run on pairs of multiprocessors
        self.tc_pair_min_rows = 256
        # grouped products with at least this many rows per group on average do too.  Measured at Scout's expert
        # shapes with 512 rows a group: 1324 against 1340 us (gate/up) and 676 against 682 us (down): what the pair
        # saves in shared-memory traffic, the part-filled last tile of 256 rows gives back.
        self.tc_pair_min_group_rows = 512
        self.skinny_tall_rows = 0
        # grouped products with at most this many rows per group on average run with the operands swapped
        self.use_tc_experts = True
        self.tc_experts_max_group_rows = 64
        self.tc_experts_down_min_groups = 64
        # the TMA weight-streaming kernel for decode products
        self.use_stream = True
        # what a work item costs besides its stages, in stages of 16 KiB: any item; one whose sums cross blocks (a
        # fence, a ticket, a second pass: about 2.7 us) and every k split of it; one whose k slices meet in shared memory
        self.stream_item_cost = 2.0
        self.stream_split_item_cost = 6.0
        self.stream_split_cost = 1.5
        self.stream_slice_cost = 1.0
        self.stream_max_slices = 8             # 1: tiles of 128 rows only
        self.stream_slices_min_rows = 6        # products of fewer rows keep tiles of 128 rows (see stream_cut)
        self.stream_slices_grouped = False     # ... and so do grouped products
        self.stream_cluster_max_rows = 3       # up to this many rows the k splits of a tile are a thread-block cluster (0: never)
        # ... if they are no more than this (the hardware takes up to 8).  Measured in the decode step at one / two /
        # three tokens: no clusters 2.780 / 3.348 / 4.114 ms, clusters of two (the gate/up products) 2.748 / 3.335 /
        # 4.079, up to four 2.749 / 3.313 / 4.082, up to eight 2.753 / 3.316 / 4.083; clusters of seven (the 40 tiles of
        # an output projection) are not all resident at once and are refused by the kernel's launcher
        self.stream_cluster_max_splits = 4
        # what such an item costs besides its stages (see stream_cut).  9 (qkv in four splits as clusters, the output
        # and down projections in seven through global memory) against 4, 2, 1 (all three in four): 2.714 against
        # 2.738, 2.727, 2.726 ms at one token
        self.stream_cluster_cost = 9.0
        # one-group products of up to this many rows stream their weights too (16: never; the kernel takes up to 32).
        # Decode step at 20 / 24 / 32 requests: 11.98 / 12.63 / 14.07 ms against 12.17 / 13.07 / 14.30 on tcgen05
        self.stream_max_rows = 32
        self.stream_force = None               # (k slices, k splits) for every call, for measurements
        # (shared memory per block, resident blocks) for up to 3 tokens and for more: measured in the decode step at
        # Scout shapes, one token 2.90 ms with (110 KiB, 2 per multiprocessor) against 3.01 with (74 KiB, 3), eight
        # tokens 7.10 against 7.02, sixty-four alike; one block per multiprocessor with 110 or 200 KiB: 3.2 and 3.1 ms
        self.stream_shape = [(110 * 1024, 2 * self.sm_count), (74 * 1024, 3 * self.sm_count)]
        # arrival counters of the splits (zero between calls), one set per stream, since calls that share a set must not
        # overlap.  The sets are made ahead: one made while a CUDA graph is captured would lie in the graphs' memory
        # pool, where a graph captured before keeps its temporaries.
        self._tickets, self._tickets_n = {}, 65536
        self._spare_tickets = [torch.zeros(self._tickets_n, dtype=torch.int32, device=self.device) for _ in range(4)]

    # ------------------------------------------------------------------ helpers
    def _tickets_of(self, stream: int):
        tickets = self._tickets.get(stream)
        if tickets is None:
            if not torch.cuda.is_current_stream_capturing():
                self._spare_tickets.append(torch.zeros(self._tickets_n, dtype=torch.int32, device=self.device))
            if not self._spare_tickets:
                raise KernelError("a graph capture on yet another stream has no arrival counters left")
            tickets = self._tickets[stream] = self._spare_tickets.pop(0)
        return tickets

    def _count(self, library, n=1):
        self.launches += n
        self.launches_by_library[library] += n

    def _lib(self, name):
        lib = self._libs.get(name)
        if lib is None:
            lib = self._libs[name] = build.load(name)
            if name in _WAITING_LIBRARIES and name not in _configured:
                word = _error_buffer().data_ptr() + 4 * _WAITING_LIBRARIES.index(name)
                _check(self._configure_waits(lib, name, 0, word, 0), f"{name}: configure_waits")
                _configured.add(name)
        return lib

    @staticmethod
    def _configure_waits(lib, name, limit_cycles, error_word, extra_tx):
        return getattr(lib, f"spite_{name}_configure_waits")(C.c_longlong(limit_cycles), C.c_void_p(error_word),
                                                             C.c_int(extra_tx))

    def configure_waits(self, library: str, *, limit_cycles: int = 0, extra_tx: int = 0):
        """Set the limit (clock cycles; 0: the default of about two seconds) of the bounded waits in
        `library`'s kernels for later launches.  `extra_tx` exists for one test: it makes the first
        barrier of every block of `gemm_tc` incomplete, so that the waits on it run out."""
        lib = self._lib(library)
        word = _error_buffer().data_ptr() + 4 * _WAITING_LIBRARIES.index(library)
        _check(self._configure_waits(lib, library, limit_cycles, word, extra_tx), f"{library}: configure_waits")

    def errors(self) -> dict:
        words = _error_buffer()
        out = {}
        for i, name in enumerate(_WAITING_LIBRARIES):
            code = int(words[i])
            if code:
                out[name] = code
                words[i] = 0
        return out

    @staticmethod
    def _stream():
        return C.c_void_p(torch.cuda.current_stream().cuda_stream)

    def _t(self, t, dtype=None, name="tensor"):
        if t.device.type != "cuda" or not t.is_contiguous():
            raise KernelError(f"{name} must be a contiguous CUDA tensor")
        if dtype is not None and t.dtype != dtype:
            raise KernelError(f"{name} must be {dtype}, is {t.dtype}")
        return t

    # ------------------------------------------------------------------ elementwise
    def embed(self, table, token_ids, out_h, *, scale=1.0, position_table=None, positions=None, copies=1):
        self._t(table, self.dtype, "table"); self._t(token_ids, torch.int32, "token_ids")
        self._t(out_h, torch.float32, "out_h")
        V, d = table.shape
        if out_h.numel() != token_ids.numel() * copies * d or (copies != 1 and position_table is not None):
            raise KernelError("embed: the output does not fit")
        if position_table is not None:
            self._t(position_table, self.dtype, "position_table"); self._t(positions, torch.int32, "positions")
            if position_table.shape[1] != d or positions.numel() != token_ids.numel():
                raise KernelError("embed: the position table or the positions do not fit")
            st = self._lib("elementwise").spite_embed_positions(
                self._dt, C.c_void_p(table.data_ptr()), C.c_void_p(token_ids.data_ptr()),
                C.c_void_p(position_table.data_ptr()), C.c_void_p(positions.data_ptr()), C.c_void_p(out_h.data_ptr()),
                token_ids.numel(), d, V, position_table.shape[0], C.c_float(scale), self._stream())
            self._count("elementwise", 1)
            _check(st, "embed (with positions)")
            return
        st = self._lib("elementwise").spite_embed(
            self._dt, C.c_void_p(table.data_ptr()), C.c_void_p(token_ids.data_ptr()),
            C.c_void_p(out_h.data_ptr()), token_ids.numel(), d, V, C.c_float(scale), int(copies), self._stream())
        self._count("elementwise", 1)
        _check(st, "embed")

    def pack_pair(self, a, b, out, *, refill=None):
        self._t(a, torch.float32, "a"); self._t(b, torch.float32, "b"); self._t(out, self.dtype, "out")
        M, d = a.shape
        if tuple(b.shape) != (M, d) or tuple(out.shape) != (M, 2 * d):
            raise KernelError("pack_pair: shapes do not fit")
        if refill is not None and (self._t(refill, torch.float32, "refill").numel() != d):
            raise KernelError("pack_pair: the refill vector must have the streams' width")
        st = self._lib("elementwise").spite_pack_pair(
            self._dt, C.c_void_p(a.data_ptr()), C.c_void_p(b.data_ptr()), C.c_void_p(_ptr(refill)),
            C.c_void_p(out.data_ptr()), M, d, self._stream())
        self._count("elementwise", 1)
        _check(st, "pack_pair")

    def transform_logits(self, logits, *, scale=1.0, softcap=None):
        self._t(logits, torch.float32, "logits")
        st = self._lib("elementwise").spite_transform_logits(
            C.c_void_p(logits.data_ptr()), C.c_longlong(logits.numel()), C.c_float(scale),
            C.c_float(softcap or 0.0), self._stream())
        self._count("elementwise", 1)
        _check(st, "transform_logits")

    def rms_norm(self, h, gain, eps, out, rows=None):
        self._t(h, torch.float32, "h"); self._t(gain, torch.float32, "gain"); self._t(out, None, "out")
        if rows is not None:
            self._t(rows, torch.int32, "rows")
        n, d = out.shape
        st = self._lib("elementwise").spite_rms_norm(
            _DT[out.dtype], C.c_void_p(h.data_ptr()), C.c_void_p(gain.data_ptr()),
            C.c_void_p(_ptr(rows)), C.c_void_p(out.data_ptr()), n, d, C.c_float(eps), self._stream())
        self._count("elementwise", 1)
        _check(st, "rms_norm")

    def rms_norm_residual(self, y, gain, eps, mult, h, *, next_gain=None, next_out=None):
        self._t(y, torch.float32, "y"); self._t(h, torch.float32, "h"); self._t(gain, torch.float32, "gain")
        M, d = h.shape
        if tuple(y.shape) != (M, d) or gain.numel() != d:
            raise KernelError("rms_norm_residual: shapes do not fit")
        if next_gain is not None and next_out is None:
            raise KernelError("rms_norm_residual: the next norm needs its output")
        if next_out is not None:
            self._t(next_out, None, "next_out")
            if next_gain is not None:
                self._t(next_gain, torch.float32, "next_gain")
            if tuple(next_out.shape) != (M, d) or (next_gain is not None and next_gain.numel() != d) or next_out.dtype not in _DT:
                raise KernelError("rms_norm_residual: the next norm's output or gain does not fit")
        st = self._lib("elementwise").spite_rms_norm_residual(
            _DT[next_out.dtype] if next_out is not None else self._dt, C.c_void_p(y.data_ptr()), C.c_void_p(gain.data_ptr()),
            C.c_void_p(h.data_ptr()), C.c_void_p(_ptr(next_gain)), C.c_void_p(_ptr(next_out)), M, d, C.c_float(eps),
            C.c_float(mult), self._stream())
        self._count("elementwise", 1)
        _check(st, "rms_norm_residual")

    def cast_rows(self, h, out):
        self._t(h, torch.float32, "h"); self._t(out, self.dtype, "out")
        if out.numel() != h.numel():
            raise KernelError("cast_rows: out must have as many elements as h")
        st = self._lib("elementwise").spite_cast_rows(self._dt, C.c_void_p(h.data_ptr()), C.c_void_p(out.data_ptr()),
                                                      C.c_longlong(h.numel()), self._stream())
        self._count("elementwise", 1)
        _check(st, "cast_rows")

    def short_conv(self, x, w, out, batch, state, *, channels, activation=None, state_offset=0, bias=None):
        self._t(x, torch.float32, "x"); self._t(w, torch.float32, "w"); self._t(out, None, "out")
        if state is None and w.shape[1] == 1:
            state = x[:1]                                       # one tap: nothing is carried, and the kernel touches no slot
        self._t(state, torch.float32, "state")
        if out.dtype not in (self.dtype, torch.float32):
            raise KernelError(f"short_conv: out must be {self.dtype} or float32")
        M = x.shape[0]
        taps = w.shape[1]
        if w.shape[0] != channels or out.shape[0] != M or out.shape[1] < channels or x.shape[1] < out.shape[1]:
            raise KernelError("short_conv: shapes do not fit")
        if bias is not None and self._t(bias, torch.float32, "bias").numel() != channels:
            raise KernelError("short_conv: one bias per channel")
        if activation not in (None, "silu"):
            raise KernelError(f"short_conv: unknown activation {activation!r}")
        slot_stride = state[0].numel()
        if state_offset < 0 or state_offset + (taps - 1) * channels > slot_stride:
            raise KernelError("short_conv: the slot cannot hold the convolution's rows")
        n_seg = batch.cu_seqlens.numel() - 1
        p = ShortConvParams(x=x.data_ptr(), x_stride=x.shape[1], w=w.data_ptr(), out=out.data_ptr(), out_stride=out.shape[1],
                            state=state.data_ptr() + 4 * int(state_offset), slot_stride=slot_stride,
                            cu_seqlens=batch.cu_seqlens.data_ptr(), slots=batch.slots.data_ptr(), n_segments=n_seg,
                            channels=int(channels), taps=int(taps), copy_columns=out.shape[1] - int(channels),
                            activation=1 if activation == "silu" else 0, max_seg_len=int(batch.max_seg_len), bias=_ptr(bias))
        st = self._lib("elementwise").spite_short_conv(_DT[out.dtype], C.byref(p), self._stream())
        self._count("elementwise", 1)
        _check(st, "short_conv")

    def fill_rows(self, out, vec, *, accumulate=False, other=None):
        self._t(out, torch.float32, "out"); self._t(vec, torch.float32, "vec")
        M, d = out.shape
        if vec.numel() != d:
            raise KernelError("fill_rows: the vector must have the rows' width")
        if other is not None and self._t(other, torch.float32, "other").shape != out.shape:
            raise KernelError("fill_rows: what is added row by row must have the output's shape")
        st = self._lib("elementwise").spite_fill_rows(C.c_void_p(out.data_ptr()), C.c_void_p(vec.data_ptr()), C.c_void_p(_ptr(other)),
                                                      M, d, int(bool(accumulate)), self._stream())
        self._count("elementwise", 1)
        _check(st, "fill_rows")

    def head_norm_gate(self, x, out, *, heads, size, gates=None, gate_column=0, gain=None, eps=None, gate_activation="sigmoid",
                       out_column=None):
        self._t(x, None, "x"); self._t(out, self.dtype, "out")
        if gate_activation not in ("sigmoid", "silu"):
            raise KernelError(f"head_norm_gate: unknown gate activation {gate_activation!r}")
        if x.dtype not in (self.dtype, torch.float32):
            raise KernelError(f"head_norm_gate: x must be {self.dtype} or float32")
        M = x.shape[0]
        if tuple(x.shape) != (M, heads * size) or (out_column is None and tuple(out.shape) != (M, heads * size)):
            raise KernelError("head_norm_gate: x and out must be [tokens, heads * size]")
        o_ptr = self._columns(out, out_column or 0, heads * size, M, "head_norm_gate: out")
        g_ptr, g_stride = None, 0
        if gates is not None:
            self._t(gates, x.dtype, "gates")
            if gates.dim() != 2 or gates.shape[0] != M or gate_column < 0 or gate_column + heads * size > gates.shape[1]:
                raise KernelError("head_norm_gate: the gate columns do not fit")
            g_ptr, g_stride = gates.data_ptr() + int(gate_column) * gates.element_size(), gates.shape[1]
        if gain is not None and self._t(gain, torch.float32, "gain").numel() not in (heads * size, size):
            raise KernelError("head_norm_gate: the gain must have heads * size elements, or a head's")
        st = self._lib("elementwise").spite_head_norm_gate(
            _DT[x.dtype], self._dt, C.c_void_p(x.data_ptr()), C.c_void_p(g_ptr), C.c_longlong(g_stride),
            C.c_void_p(_ptr(gain)), C.c_void_p(o_ptr), C.c_longlong(out.shape[1]), M, int(heads), int(size), C.c_float(eps or 0.0),
            int(gate_activation == "silu"), int(gain is not None and gain.numel() == heads * size), self._stream())
        self._count("elementwise", 1)
        _check(st, "head_norm_gate")

    @staticmethod
    def _columns(t, column, width, rows, what):
        """Address of column `column` of the 2-D tensor `t`, whose rows must have `width` columns from there on."""
        if t.dim() != 2 or t.shape[0] != rows or column < 0 or column + width > t.shape[1]:
            raise KernelError(f"{what} must be [tokens, *] with {width} columns from column {column} on")
        return t.data_ptr() + int(column) * t.element_size()

    def token_shift(self, x, mu, out, batch, state, *, state_offset=0, offsets_out=None):
        self._t(x, self.dtype, "x"); self._t(mu, torch.float32, "mu"); self._t(out, self.dtype, "out")
        self._t(state, torch.float32, "state")
        M, d = x.shape
        n = mu.shape[0]
        slot_stride = state[0].numel()
        if mu.shape[1] != d or tuple(out.shape) != (n, M, d) or state_offset < 0 or state_offset + d > slot_stride:
            raise KernelError("token_shift: shapes do not fit")
        if offsets_out is not None and self._t(offsets_out, torch.int32, "offsets_out").numel() != n + 1:
            raise KernelError("token_shift: one offset per mix and one behind them")
        p = TokenShiftParams(x=x.data_ptr(), mu=mu.data_ptr(), out=out.data_ptr(), state=state.data_ptr() + 4 * int(state_offset),
                             slot_stride=slot_stride, seg_of_token=batch.seg_of_token.data_ptr(),
                             cu_seqlens=batch.cu_seqlens.data_ptr(), slots=batch.slots.data_ptr(), offsets_out=_ptr(offsets_out),
                             n_tokens=M, d=d, n_mixes=n)
        st = self._lib("elementwise").spite_token_shift(self._dt, C.byref(p), self._stream())
        self._count("elementwise", 1)
        _check(st, "token_shift")

    def gate_group_norm(self, x, z, gain, out, *, groups, eps, z_column=0):
        self._t(x, torch.float32, "x"); self._t(z, torch.float32, "z"); self._t(gain, torch.float32, "gain")
        self._t(out, self.dtype, "out")
        M, n = x.shape
        if n % groups or tuple(out.shape) != (M, n) or gain.numel() != n:
            raise KernelError("gate_group_norm: shapes do not fit")
        z_ptr = self._columns(z, z_column, n, M, "gate_group_norm: z")
        st = self._lib("elementwise").spite_gate_group_norm(
            self._dt, C.c_void_p(x.data_ptr()), C.c_void_p(z_ptr), C.c_longlong(z.shape[1]), C.c_void_p(gain.data_ptr()),
            C.c_void_p(out.data_ptr()), M, int(groups), n // int(groups), C.c_float(eps), self._stream())
        self._count("elementwise", 1)
        _check(st, "gate_group_norm")

    def streams(self, x, *, y=None, bias=None, scale=None, mix=None, w_out=None, w_in=None, gain=None, eps=None, next_out=None,
                rows=None, write_back=True):
        self._t(x, torch.float32, "x")
        M, n, d = x.shape
        for name, t, numel in (("y", y, M * d), ("bias", bias, d), ("scale", scale, d), ("mix", mix, n * n), ("w_out", w_out, n),
                               ("w_in", w_in, n), ("gain", gain, d)):
            if t is not None and self._t(t, torch.float32, name).numel() != numel:
                raise KernelError(f"streams: {name} has {t.numel()} elements, {numel} are needed")
        R = M
        if rows is not None:
            R = self._t(rows, torch.int32, "rows").numel()
        if next_out is not None and (next_out.dtype not in _DT or tuple(self._t(next_out, None, "next_out").shape) != (R, d)):
            raise KernelError("streams: next_out must be [rows, width]")
        p = StreamsParams(x=x.data_ptr(), y=_ptr(y), bias=_ptr(bias), scale=_ptr(scale), mix=_ptr(mix), w_out=_ptr(w_out),
                          w_in=_ptr(w_in), gain=_ptr(gain), next_out=_ptr(next_out), rows=_ptr(rows), n_rows=R, d=d, streams=n,
                          write_back=int(bool(write_back)), eps=float(eps or 0.0))
        st = self._lib("elementwise").spite_streams(_DT[next_out.dtype] if next_out is not None else 0, C.byref(p), self._stream())
        self._count("elementwise", 1)
        _check(st, "streams")

    def clear_pages(self, kv, page_ids):
        self._t(kv, None, "cache")
        if not page_ids:
            return
        caches, two, pages = kv.shape[0], kv.shape[1], kv.shape[2]
        page_bytes = kv.stride(2) * kv.element_size()
        ids = (C.c_int * len(page_ids))(*page_ids)
        st = self._lib("elementwise").spite_clear_pages(
            C.c_void_p(kv.data_ptr()), C.c_longlong(caches * two), C.c_longlong(kv.stride(1) * kv.element_size()),
            C.c_longlong(page_bytes), pages, ids, len(page_ids), self._stream())
        self._count("elementwise", -(-len(page_ids) // 60))
        _check(st, "clear_pages")

    # ------------------------------------------------------------------ matrix products
    def _gemm(self, p: GemmParams, what, max_rows_per_group, gather_src=None, even_groups=False):
        """Pick the kernel.  bfloat16: up to 16 rows (a decode step) go to the TMA weight-streaming
        kernel when K is a multiple of 64, else to the register-ring streaming kernel; more rows to
        the tcgen05 kernels (TMA-fed, accumulators in TMEM): one group of 256 rows and more, or groups
        of 512 rows on average, on pairs of multiprocessors, the rest on one block a tile; a very
        tall matrix (output head) goes there even with few rows.  float32, and shapes those refuse, go to the CUDA-core kernel.
        `gather_src` is the tensor whose rows `p.a_rows` gathers: the tcgen05 kernel wants contiguous
        rows, so they are gathered first.  `even_groups`: every group has `max_rows_per_group` rows."""
        if self.dtype == torch.bfloat16:
            grouped = bool(p.group_offsets)
            # measured on B200 at Scout shapes: the streaming kernel wins up to 16 rows except on very
            # tall matrices (output head), where the TMA pipeline of the tcgen05 kernel streams better
            few = (max_rows_per_group if even_groups else p.M) <= self.skinny_max_rows and not (not grouped and p.N >= 65536 and p.M > self.skinny_tall_rows)
            tc_ok = self.use_tcgen05 and p.K % 8 == 0 and p.lda % 8 == 0
            # ... and a one-group product of up to 32 rows in place (the dense projections of a larger decode batch)
            more = (not grouped and not p.a_rows and 16 < p.M <= self.stream_max_rows and p.N < 65536)
            if (few or more) and self.use_stream and p.K % 64 == 0 and max_rows_per_group <= (32 if more else 16):
                st = self._gemm_stream(p, int(max_rows_per_group), grouped, int(max_rows_per_group) if even_groups else p.M)
                if st != -2:
                    self._count("gemm_stream", 1)
                    _check(st, what + " (streaming)")
                    return
            if few or (not tc_ok and max_rows_per_group <= 64):
                st = self._lib("gemm_skinny").spite_gemm_skinny(C.byref(p), int(max_rows_per_group), self.skinny_blocks,
                                                                self._stream())
                if st != -2:                       # -2: shape outside the kernel's domain, fall through
                    self._count("gemm_skinny", 1)
                    _check(st, what)
                    return
            if tc_ok:
                orig = p
                if gather_src is not None:
                    keep = torch.empty_like(gather_src)
                    st = self._lib("elementwise").spite_gather_rows(
                        C.c_void_p(gather_src.data_ptr()), C.c_void_p(p.a_rows), C.c_void_p(keep.data_ptr()),
                        gather_src.shape[0], C.c_longlong(gather_src.shape[1] * gather_src.element_size()),
                        self._stream())
                    self._count("elementwise", 1)
                    _check(st, "gather_rows")
                    p = GemmParams.from_buffer_copy(p)
                    p.A = keep.data_ptr()          # rows are in place now; a_rows only indexes the row scale
                if grouped and self.use_tc_experts and self._few_rows_per_group(p):
                    # groups of few rows each (experts of a prompt portion): the weights as the 128-row operand, a
                    # group's tokens as the instruction's columns
                    st = self._lib("gemm_tc_experts").spite_gemm_tc_experts(C.byref(p), self.sm_count, self._stream())
                    if st != -2:
                        self._count("gemm_tc_experts", 1)
                        _check(st, what + " (tcgen05, experts)")
                        return
                if p.M >= (self.tc_pair_min_group_rows * p.n_groups if grouped else self.tc_pair_min_rows):
                    # a product of many rows (per group) on pairs of multiprocessors (tcgen05 cta_group::2)
                    st = self._lib("gemm_tc_pair").spite_gemm_tc_pair(C.byref(p), self.sm_count // 2, self._stream())
                    if st != -2:
                        self._count("gemm_tc_pair", 1)
                        _check(st, what + " (tcgen05, pairs)")
                        return
                st = self._lib("gemm_tc").spite_gemm_tc(C.byref(p), self.sm_count, self._stream())
                if st != -2:
                    self._count("gemm_tc", 1)
                    _check(st, what + " (tcgen05)")
                    return
                p = orig
                if max_rows_per_group <= 64:       # refused (alignment): the streaming kernel may still take it
                    st = self._lib("gemm_skinny").spite_gemm_skinny(C.byref(p), int(max_rows_per_group),
                                                                    self.skinny_blocks, self._stream())
                    if st != -2:
                        self._count("gemm_skinny", 1)
                        _check(st, what)
                        return
        st = self._lib("gemm_simt").spite_gemm_simt(self._dt, C.byref(p), self._stream())
        self._count("gemm_simt", 1)
        _check(st, what)

    def _few_rows_per_group(self, p) -> bool:
        """Does a grouped product go to the kernel with swapped operands?  Measured on B200 at Scout's expert
        shapes (us, swapped against 128-row tiles).  Gate/up with SwiGLU, 16 experts: 427/437 at 256 tokens,
        437/464 at 1,024, 630/503 at 2,048 (half the groups then exceed a token tile and run twice); 128
        experts: 3,159/3,300 at 1,024, 3,284/3,849 at 8,192.  Down product into the residual stream, 16
        experts: 264/244 at 256, 276/254 at 1,024, 344/293 at 2,048; 128 experts: 1,749/1,705 at 2,048,
        1,905/2,006 at 8,192.  So: gate/up up to 64 rows a group on average, the down product only with
        many groups of 32 to 64 rows."""
        avg = p.M / p.n_groups
        if p.epilogue == EPI_SWIGLU or (p.epilogue == EPI_STORE and p.row_scale):     # an expert's first product
            return avg <= self.tc_experts_max_group_rows
        if p.epilogue == EPI_ADD_F32:
            return p.n_groups >= self.tc_experts_down_min_groups and 32 <= avg <= self.tc_experts_max_group_rows
        return False

    def _gemm_stream(self, p, max_rows_per_group, grouped, rows):
        """The TMA weight-streaming kernel for decode steps: picks the tile height (k slices inside the block)
        and the k splits across blocks so that the work items are many enough to spread evenly, and lends the
        scratch for the partial sums of the splits."""
        swiglu = p.epilogue == EPI_SWIGLU
        groups = min(p.n_groups, p.M) if grouped else 1
        smem, blocks = self.stream_shape[0 if rows <= 3 or rows > 16 else 1]      # (the tokens of many rows need the larger ring)
        nt = 8 if max_rows_per_group <= 8 else 16 if max_rows_per_group <= 16 else 32
        slices, splits = self.stream_force or self._stream_cut(rows, p.N, p.K, groups, swiglu, blocks, smem, nt, grouped)
        tile_rows = 128 // slices
        tiles = -(-p.N // (tile_rows // 2 if swiglu else tile_rows)) * groups
        lib = self._lib("gemm_stream")
        stream = torch.cuda.current_stream().cuda_stream
        if slices == 1 and 2 <= splits <= self.stream_cluster_max_splits and rows <= self.stream_cluster_max_rows:
            # the k splits of a tile as one thread-block cluster: their sums meet in shared memory
            st = lib.spite_gemm_stream(C.byref(p), max_rows_per_group, 1, 1, blocks, smem, splits, None, C.c_longlong(0),
                                       None, 0, C.c_void_p(stream))
            if st != -2:
                return st
        scratch, n_floats = None, 0
        if splits > 1:
            if tiles > self._tickets_n:
                return -2
            n_floats = tiles * splits * nt * tile_rows
            scratch = torch.empty(n_floats, dtype=torch.float32, device=self.device)
        tickets = self._tickets_of(stream) if splits > 1 else None
        return lib.spite_gemm_stream(
            C.byref(p), max_rows_per_group, slices, 0, blocks, smem, splits, C.c_void_p(_ptr(scratch)),
            C.c_longlong(n_floats), C.c_void_p(_ptr(tickets)), self._tickets_n, C.c_void_p(stream))

    def _stream_cut(self, M: int, N: int, K: int, groups: int, swiglu: bool, slots: int, smem: int, nt: int,
                    grouped: bool):
        return stream_cut(M, N, K, groups, swiglu, slots, smem, nt, item_cost=self.stream_item_cost,
                          split_item_cost=self.stream_split_item_cost, split_cost=self.stream_split_cost,
                          slice_cost=self.stream_slice_cost,
                          max_slices=(min(2, self.stream_max_slices) if nt > 16 else self.stream_max_slices)
                          if self.stream_slices_grouped or not grouped else 1,
                          slices_min_rows=self.stream_slices_min_rows,
                          cluster_max_splits=self.stream_cluster_max_splits if M <= self.stream_cluster_max_rows else 0,
                          cluster_cost=self.stream_cluster_cost)

    def attention_tc_error(self) -> int:
        """Error code left by a tcgen05 attention block that gave up waiting (0: none); clears it. Synchronises."""
        torch.cuda.synchronize(self.device)
        words = _error_buffer()
        code, words[3] = int(words[3]), 0
        return code

    def gemm_tc_error(self) -> int:
        """Error code left by a product kernel's block that gave up waiting (0: none); clears it. Synchronises."""
        torch.cuda.synchronize(self.device)
        words = _error_buffer()
        code = int(words[0]) or int(words[1]) or int(words[2]) or int(words[5])
        words[:3] = 0
        words[5] = 0
        return code

    def linear(self, x, w, out, *, accumulate=False, row_scale=None, activation=None, bias=None, act_params=None):
        self._t(x, self.dtype, "x"); self._t(w, self.dtype, "w"); self._t(out, None, "out")
        M, K = x.shape
        N = w.shape[0]
        if w.shape[1] != K or tuple(out.shape) != (M, N):
            raise KernelError(f"linear: x {tuple(x.shape)}, w {tuple(w.shape)}, out {tuple(out.shape)} do not fit")
        if accumulate:
            if out.dtype != torch.float32:
                raise KernelError("linear(accumulate=True) needs a float32 output")
            epi = EPI_ADD_F32
        elif out.dtype == torch.float32 and self.dtype != torch.float32:
            epi = EPI_STORE_F32
        elif out.dtype == self.dtype:
            epi = EPI_STORE
        else:
            raise KernelError(f"linear: output type {out.dtype} not supported")
        if activation not in _ACTIVATION or (activation is not None and epi != EPI_STORE):
            raise KernelError(f"linear: activation {activation!r} needs a plain store in the activation type")
        if bias is not None and (epi != EPI_STORE or self._t(bias, torch.float32, "bias").numel() != N):
            raise KernelError("linear: a bias goes with a plain store and has one element per output column")
        if (activation == "xielu") != (act_params is not None):
            raise KernelError("linear: act_params are the two coefficients of the activation 'xielu'")
        pos, neg = act_params or (0.0, 0.0)
        p = GemmParams(A=x.data_ptr(), W=w.data_ptr(), C=out.data_ptr(), a_rows=None, c_rows=None,
                       group_offsets=None, row_scale=_ptr(row_scale), lda=K, ldc=N, w_group_stride=0,
                       n_groups=1, M=M, N=N, K=K, epilogue=epi, scale_by_a_row=0, activation=_ACTIVATION[activation],
                       bias=_ptr(bias), act_pos=float(pos), act_neg=float(neg))
        self._gemm(p, "linear", M)

    def linear_swiglu(self, x, w_gate_up, out, *, row_scale=None, activation="silu"):
        self._t(x, self.dtype, "x"); self._t(w_gate_up, self.dtype, "w"); self._t(out, self.dtype, "out")
        M, K = x.shape
        F = w_gate_up.shape[0] // 2
        if w_gate_up.shape != (2 * F, K) or tuple(out.shape) != (M, F):
            raise KernelError("linear_swiglu: shapes do not fit")
        if activation not in ("silu", "gelu_tanh"):
            raise KernelError(f"linear_swiglu: unknown gate function {activation!r}")
        p = GemmParams(A=x.data_ptr(), W=w_gate_up.data_ptr(), C=out.data_ptr(), a_rows=None, c_rows=None,
                       group_offsets=None, row_scale=_ptr(row_scale), lda=K, ldc=F, w_group_stride=0,
                       n_groups=1, M=M, N=F, K=K, epilogue=EPI_SWIGLU, scale_by_a_row=0,
                       activation=0 if activation == "silu" else _ACTIVATION[activation])
        self._gemm(p, "linear_swiglu", M)

    def grouped_linear_swiglu(self, x, w_gate_up, sorted_rows, offsets, row_scale, out):
        self._t(x, self.dtype, "x"); self._t(w_gate_up, self.dtype, "w"); self._t(out, self.dtype, "out")
        self._t(sorted_rows, torch.int32, "sorted_rows"); self._t(offsets, torch.int32, "offsets")
        M, K = x.shape
        E, F2, K2 = w_gate_up.shape
        F = F2 // 2
        if K2 != K or tuple(out.shape) != (M, F) or offsets.numel() != E + 1 or sorted_rows.numel() != M:
            raise KernelError("grouped_linear_swiglu: shapes do not fit")
        p = GemmParams(A=x.data_ptr(), W=w_gate_up.data_ptr(), C=out.data_ptr(),
                       a_rows=sorted_rows.data_ptr(), c_rows=None, group_offsets=offsets.data_ptr(),
                       row_scale=_ptr(row_scale), lda=K, ldc=F, w_group_stride=F2 * K,
                       n_groups=E, M=M, N=F, K=K, epilogue=EPI_SWIGLU, scale_by_a_row=1)
        self._gemm(p, "grouped_linear_swiglu", M, gather_src=x)

    def grouped_linear_act(self, x, w_up, sorted_rows, offsets, row_scale, out, *, activation="relu2"):
        self._t(x, self.dtype, "x"); self._t(w_up, self.dtype, "w"); self._t(out, self.dtype, "out")
        self._t(sorted_rows, torch.int32, "sorted_rows"); self._t(offsets, torch.int32, "offsets")
        M, K = x.shape
        E, F, K2 = w_up.shape
        if K2 != K or tuple(out.shape) != (M, F) or offsets.numel() != E + 1 or sorted_rows.numel() != M:
            raise KernelError("grouped_linear_act: shapes do not fit")
        if activation not in _ACTIVATION:
            raise KernelError(f"grouped_linear_act: unknown activation {activation!r}")
        p = GemmParams(A=x.data_ptr(), W=w_up.data_ptr(), C=out.data_ptr(),
                       a_rows=sorted_rows.data_ptr(), c_rows=None, group_offsets=offsets.data_ptr(),
                       row_scale=_ptr(row_scale), lda=K, ldc=F, w_group_stride=F * K,
                       n_groups=E, M=M, N=F, K=K, epilogue=EPI_STORE, scale_by_a_row=1,
                       activation=_ACTIVATION[activation])
        self._gemm(p, "grouped_linear_act", M, gather_src=x)

    def grouped_linear_accumulate(self, a, w_down, sorted_rows, offsets, h, *, row_scale=None):
        self._t(a, self.dtype, "a"); self._t(w_down, self.dtype, "w"); self._t(h, torch.float32, "h")
        if row_scale is not None and self._t(row_scale, torch.float32, "row_scale").numel() != a.shape[0]:
            raise KernelError("grouped_linear_accumulate: one scale per row of the sorted order")
        M, F = a.shape
        E, d, F2 = w_down.shape
        if F2 != F or h.shape[1] != d or offsets.numel() != E + 1 or sorted_rows.numel() != M:
            raise KernelError("grouped_linear_accumulate: shapes do not fit")
        p = GemmParams(A=a.data_ptr(), W=w_down.data_ptr(), C=h.data_ptr(), a_rows=None,
                       c_rows=sorted_rows.data_ptr(), group_offsets=offsets.data_ptr(), row_scale=_ptr(row_scale),
                       lda=F, ldc=d, w_group_stride=d * F, n_groups=E, M=M, N=d, K=F,
                       epilogue=EPI_ADD_F32, scale_by_a_row=0)
        self._gemm(p, "grouped_linear_accumulate", M)

    def grouped_linear_rows(self, a, w, rows, offsets, out, *, a_sorted=False):
        self._t(a, self.dtype, "a"); self._t(w, self.dtype, "w"); self._t(out, self.dtype, "out")
        self._t(rows, torch.int32, "rows"); self._t(offsets, torch.int32, "offsets")
        R, lda = a.shape
        G, N, K = w.shape
        M = rows.numel()
        if K > lda or (a.shape[0] != M if a_sorted else out.shape[0] != R) or N > out.shape[1] or offsets.numel() != G + 1 \
                or M > out.shape[0]:
            raise KernelError("grouped_linear_rows: shapes do not fit")
        # the rows are gathered and scattered by the same list (or only scattered, if `a` lies in the list's order already);
        # columns beyond K of `a` and beyond N of `out` stay out
        p = GemmParams(A=a.data_ptr(), W=w.data_ptr(), C=out.data_ptr(), a_rows=None if a_sorted else rows.data_ptr(),
                       c_rows=rows.data_ptr(), group_offsets=offsets.data_ptr(), row_scale=None, lda=lda, ldc=out.shape[1],
                       w_group_stride=N * K, n_groups=G, M=M, N=N, K=K, epilogue=EPI_STORE, scale_by_a_row=0)
        self._gemm(p, "grouped_linear_rows", M, gather_src=None if a_sorted else a)

    def batched_linear(self, x, w, offsets, out):
        self._t(x, self.dtype, "x"); self._t(w, self.dtype, "w"); self._t(out, torch.float32, "out")
        self._t(offsets, torch.int32, "offsets")
        G, M, K = x.shape
        N = w.shape[1]
        if w.shape[0] != G or w.shape[2] != K or tuple(out.shape) != (G, M, N) or offsets.numel() != G + 1:
            raise KernelError("batched_linear: shapes do not fit")
        p = GemmParams(A=x.data_ptr(), W=w.data_ptr(), C=out.data_ptr(), a_rows=None, c_rows=None,
                       group_offsets=offsets.data_ptr(), row_scale=None, lda=K, ldc=N, w_group_stride=N * K,
                       n_groups=G, M=G * M, N=N, K=K, epilogue=EPI_STORE_F32, scale_by_a_row=0)
        self._gemm(p, "batched_linear", M, even_groups=True)

    # ------------------------------------------------------------------ attention
    def _step_tokens(self, batch, group):
        bt = batch.block_tables[group]
        return StepTokens(positions=batch.positions.data_ptr(), seg_of_token=batch.seg_of_token.data_ptr(),
                          block_table=bt.data_ptr(), table_width=bt.shape[1], n_tokens=batch.n_tokens)

    def _paged(self, cache):
        kv = cache.kv                       # [planes, pages, nkv, page_size, hd]; one plane: the key rows are the values
        self._t(kv, self.dtype, "cache")
        if cache.key_scale is not None and tuple(self._t(cache.key_scale, torch.float32, "key_scale").shape) != tuple(kv.shape[1:4]):
            raise KernelError("a cache's key factors are [pages, kv heads, page_size]")
        return PagedCache(key_scale=_ptr(cache.key_scale), kv=kv.data_ptr(), v_offset=kv.stride(0) if kv.shape[0] == 2 else 0, n_pages=kv.shape[1],
                          page_size=kv.shape[3], num_kv_heads=kv.shape[2], head_dim=kv.shape[4])

    def qk_prepare(self, qkv, q_out, batch, cache, *, num_heads, rotation, qk_norm, temperature,
                   value_mix=None, gates_out=None, bias=None, q_only=False, norm_dim=None, value_rotation=None,
                   values_are_keys=False):
        self._t(qkv, self.dtype, "qkv"); self._t(q_out, self.dtype, "q_out")
        head_dim = cache.kv.shape[4]
        if values_are_keys and (q_only or value_mix is not None or value_rotation is not None or rotation is not None
                                or (qk_norm is not None and qk_norm.k_gain is not None)):
            raise KernelError("qk_prepare: values that are the keys are neither borrowed, blended nor rotated, their norm has no gain")
        n_cols = (num_heads + (0 if q_only else (1 if values_are_keys else 2) * cache.kv.shape[2])) * head_dim
        if qkv.shape[1] < n_cols:
            raise KernelError(f"qk_prepare: rows of {qkv.shape[1]} elements cannot hold the heads' {n_cols}")
        if bias is not None and self._t(bias, torch.float32, "bias").numel() != n_cols:
            raise KernelError(f"qk_prepare: the bias has {bias.numel()} elements, the heads have {n_cols}")
        if q_only and cache.write:
            raise KernelError("qk_prepare: a layer without keys and values of its own cannot append to the cache")
        if cache.kv.shape[0] != (1 if values_are_keys else 2) or values_are_keys != (cache.key_scale is not None):
            raise KernelError("qk_prepare appends keys and values: the cache needs both planes; keys that are the values need one, "
                              "and a factor per key")
        inv_freq, pairing, rotary_dim, amplitude = None, 0, head_dim, 1.0
        v_other, v_stride, v_head, v_dim, v_lam = None, 0, 0, 0, 0.0
        if value_mix is not None:
            other, column, v_head, v_dim, v_lam = value_mix
            self._t(other, self.dtype, "value_mix source")
            if other.shape[0] != qkv.shape[0]:
                raise KernelError("qk_prepare: the values to blend in belong to other tokens")
            v_other, v_stride = other.data_ptr() + int(column) * other.element_size(), other.shape[1]
        if gates_out is not None:
            self._t(gates_out, torch.float32, "gates_out")
            if tuple(gates_out.shape) != (qkv.shape[0], num_heads):
                raise KernelError("qk_prepare: gates_out must be [tokens, heads]")
        if rotation is not None:
            amplitude = float(rotation.amplitude)
            inv_freq = self._t(rotation.inv_freq, torch.float32, "inv_freq")
            pairing = {"neighbours": 0, "halves": 1}[rotation.pairing]
            rotary_dim = int(rotation.rotary_dim or head_dim)
            if inv_freq.numel() != rotary_dim // 2:
                raise KernelError(f"qk_prepare: {inv_freq.numel()} frequencies for {rotary_dim} rotating elements")
        v_freq, v_dims, v_pairing, v_low = None, 0, 0, None
        low = self._freq_low(rotation)
        if value_rotation is not None:
            f = self._t(value_rotation.inv_freq, torch.float32, "inv_freq")
            v_freq, v_dims, v_pairing = f.data_ptr(), 2 * f.numel(), self._PAIRING[value_rotation.pairing]
            v_low = self._freq_low(value_rotation)
            if value_rotation.amplitude != 1.0 or (value_rotation.rotary_dim or v_dims) != v_dims:
                raise KernelError("qk_prepare: values turn by a pure rotation")
        eps, before, q_gain, k_gain = 0.0, 0, None, None
        if qk_norm is not None:
            eps, before = float(qk_norm.eps), int(qk_norm.before_rotation)
            for g in (qk_norm.q_gain, qk_norm.k_gain):
                if g is not None and (self._t(g, torch.float32, "gain").numel() != head_dim):
                    raise KernelError("qk_prepare: a gain vector must have head_dim elements")
            q_gain, k_gain = qk_norm.q_gain, qk_norm.k_gain
        floor, scale = (int(temperature[0]), float(temperature[1])) if temperature else (0, 0.0)
        p = QkPrepareParams(qkv=qkv.data_ptr(), q_out=q_out.data_ptr(), inv_freq=_ptr(inv_freq),
                            q_gain=_ptr(q_gain), k_gain=_ptr(k_gain), qk_norm_eps=eps,
                            norm_before_rotation=before, pairing=pairing, rotary_dim=rotary_dim,
                            temperature_floor=floor, temperature_scale=scale, num_heads=num_heads,
                            write_cache=int(cache.write), qkv_stride=qkv.shape[1], rot_amplitude=amplitude,
                            v_other=v_other, v_other_stride=v_stride, v_other_head=int(v_head), v_mix_dim=int(v_dim),
                            v_mix=float(v_lam), gates_out=_ptr(gates_out), bias=_ptr(bias), q_only=int(bool(q_only)),
                            norm_dim=int(norm_dim or 0), v_inv_freq=v_freq, v_rotary_dim=v_dims, v_pairing=v_pairing,
                            inv_freq_low=low, v_inv_freq_low=v_low, values_are_keys=int(bool(values_are_keys)))
        b, c = self._step_tokens(batch, cache.group), self._paged(cache)
        st = self._lib("attention").spite_qk_prepare(self._dt, C.byref(p), C.byref(b), C.byref(c), self._stream())
        self._count("attention", 1)
        _check(st, "qk_prepare")

    _PAIRING = {"neighbours": 0, "halves": 1}

    def _freq_low(self, rotation):
        if rotation is None or rotation.inv_freq_low is None:
            return None
        if self._t(rotation.inv_freq_low, torch.float32, "inv_freq_low").numel() != rotation.inv_freq.numel():
            raise KernelError("a rotation's inv_freq_low must have one element per frequency")
        return rotation.inv_freq_low.data_ptr()

    def turn_heads(self, x, out, batch, *, heads, size, rotation=None, scale=1.0, out_column=0):
        self._t(x, self.dtype, "x"); self._t(out, self.dtype, "out")
        M = x.shape[0]
        if x.shape[1] % heads or x.shape[1] // heads < size:
            raise KernelError("turn_heads: x must be [tokens, heads * head_dim] with head_dim >= size")
        o_ptr = self._columns(out, out_column, heads * size, M, "turn_heads: out")
        freq, dims, pairing = None, 0, 0
        if rotation is not None:
            freq = self._t(rotation.inv_freq, torch.float32, "inv_freq")
            dims, pairing = 2 * freq.numel(), self._PAIRING[rotation.pairing]
            if rotation.amplitude != 1.0:
                raise KernelError("turn_heads: heads turn back by a pure rotation")
        st = self._lib("attention").spite_turn_heads(
            self._dt, C.c_void_p(x.data_ptr()), C.c_void_p(o_ptr), C.c_longlong(out.shape[1]),
            C.c_void_p(batch.positions.data_ptr()), C.c_void_p(_ptr(freq)), C.c_void_p(self._freq_low(rotation)), int(dims), pairing, M, int(heads),
            x.shape[1] // heads, int(size), C.c_float(scale), self._stream())
        self._count("attention", 1)
        _check(st, "turn_heads")

    def paged_attention(self, q, out, batch, cache, *, num_heads, window, softmax_scale, cache_settled=False,
                        sink_logit=None, head_sinks=None, head_slopes=None, head_gates=None, out_by_head=False,
                        score_softcap=None, distance_bias=None):
        self._t(q, self.dtype, "q"); self._t(out, self.dtype, "out")
        if score_softcap is not None and not score_softcap > 0:
            raise KernelError("paged_attention: the cap of the scores must be positive")
        if out.numel() != q.numel():
            raise KernelError("paged_attention: out must have as many elements as q")
        for name, t, n in (("head_sinks", head_sinks, num_heads), ("head_slopes", head_slopes, num_heads),
                           ("head_gates", head_gates, q.shape[0] * num_heads)):
            if t is not None and self._t(t, torch.float32, name).numel() != n:
                raise KernelError(f"paged_attention: {name} has {t.numel()} elements, {n} are needed")
        if not softmax_scale > 0:
            raise KernelError("paged_attention: the score scale must be positive")
        if distance_bias is not None:
            self._t(distance_bias.runs, torch.int32, "distance_bias.runs")
            if tuple(self._t(distance_bias.padded, torch.float32, "distance_bias.padded").shape) != \
                    (num_heads, distance_bias.length + 2 * distance_bias.PAD):
                raise KernelError("paged_attention: one row of numbers by distance per head")
        p = AttentionParams(q=q.data_ptr(), out=out.data_ptr(), num_heads=num_heads,
                            window_kind=_WINDOW[window.kind], window_size=int(window.size),
                            softmax_scale=float(softmax_scale),
                            has_sink=int(sink_logit is not None or head_sinks is not None),
                            sink_logit=float(sink_logit or 0.0), head_sinks=_ptr(head_sinks),
                            head_slopes=_ptr(head_slopes), head_gates=_ptr(head_gates),
                            out_by_head_tokens=q.shape[0] if out_by_head else 0, score_softcap=float(score_softcap or 0.0))
        if distance_bias is not None:
            p.distance_bias, p.distance_runs = distance_bias.padded.data_ptr(), distance_bias.runs.data_ptr()
            p.distance_len = distance_bias.length
        b, c = self._step_tokens(batch, cache.group), self._paged(cache)
        group = num_heads // c.num_kv_heads
        if (self.dtype == torch.bfloat16 and c.head_dim % 16 == 0 and c.head_dim <= 128 and group <= 16
                and c.page_size % 16 == 0 and batch.segments):
            # Tensor-core kernels; rows are (token, head of a kv group) pairs.  Segments of many
            # tokens (prompt portions) go to the kernel with 64 rows a block and warps that own
            # rows; segments of few tokens (decode) to the kernel with 16 rows a block whose
            # warps and blocks split the keys.
            big_from = -(-32 // group) if c.page_size % 32 == 0 else 1 << 30
            tpb, tpb_rows, tpb_tc = max(1, 16 // group), max(1, 64 // group), max(1, 128 // group)
            # tcgen05 kernel (two tiles of 128 rows a block): head sizes 64 and 128, pages of a multiple of 64 keys
            tc_from = 1 << 30
            if c.head_dim in (64, 128) and c.page_size % 64 == 0 and self.use_tcgen05_attention:
                tc_from = max(big_from, self.attention_tc_min_tokens or tpb_tc)
            n_small = n_big = n_tc = 0
            longest = 1
            for s in batch.segments:
                if s.n_tokens >= tc_from:
                    n_tc += -(-s.n_tokens // (2 * tpb_tc))        # a block serves two tiles of 128 rows
                    continue
                if s.n_tokens >= big_from:
                    n_big += -(-s.n_tokens // tpb_rows)
                    continue
                n_small += -(-s.n_tokens // tpb)
                last = s.start_pos + s.n_tokens - 1
                longest = max(longest, last - window.lowest_visible(max(s.start_pos, last - tpb + 1)) + 1)
            if n_tc:
                x = AttnMmaExtra(cu_seqlens=batch.cu_seqlens.data_ptr(), o_part=None, ml_part=None,
                                 n_segments=len(batch.segments), tokens_per_block=tpb_tc, n_splits=1,
                                 seg_min_tokens=tc_from, seg_max_tokens=0x7fffffff)
                st = self._lib("attention_tc").spite_paged_attention_tc(
                    C.byref(p), C.byref(b), C.byref(c), C.byref(x), n_tc, self.sm_count, self._stream())
                self._count("attention_tc", 1)
                _check(st, "paged_attention (tcgen05, prompt portions)")
            if n_big:
                x = AttnMmaExtra(cu_seqlens=batch.cu_seqlens.data_ptr(), o_part=None, ml_part=None,
                                 n_segments=len(batch.segments), tokens_per_block=tpb_rows, n_splits=1,
                                 seg_min_tokens=big_from, seg_max_tokens=tc_from - 1)
                st = self._lib("attention_rows").spite_paged_attention_rows(
                    C.byref(p), C.byref(b), C.byref(c), C.byref(x), n_big, self._stream())
                self._count("attention_rows", 1)
                _check(st, "paged_attention (tensor cores, prompt portions)")
            if not n_small:
                return
            if batch.context_bucket:            # fixed launch shape for a captured step
                longest = batch.context_bucket if window.kind == "full" else min(batch.context_bucket, window.size)
            if c.head_dim in (64, 128) and c.page_size % 64 == 0 and self.use_decode_attention:
                if group <= self.attention_narrow_rows and all(seg.n_tokens == 1 for seg in batch.segments if seg.n_tokens < big_from):
                    tpb = 1                     # one token a block: up to eight rows, the kernel's narrow form
                self._attention_decode(p, b, c, batch, n_small, tpb, big_from - 1, longest, num_heads, cache_settled)
                return
            tiles = -(-longest // 16) + 1
            base = n_small * c.num_kv_heads
            # key splits: fill the resident blocks (three per multiprocessor) once if the step is
            # small, else pick the split count whose last wave is fullest
            slots = 3 * self.sm_count
            if base <= slots:
                splits = slots // base
            elif base >= 4 * slots:
                splits = 1
            else:
                splits = max(range(1, 5), key=lambda s: (base * s / slots) / -(-base * s // slots))
            splits = max(1, min(splits, tiles // 8, self.attention_max_splits, 32))
            o_part = ml_part = None
            if splits > 1:
                # one row per token place of this kernel's blocks: tokens of longer segments take none
                o_part = torch.empty((n_small * tpb, num_heads, splits, c.head_dim), dtype=torch.float32,
                                     device=q.device)
                ml_part = torch.empty((n_small * tpb, num_heads, splits, 2), dtype=torch.float32, device=q.device)
                self.attention_scratch_bytes = (o_part.numel() + ml_part.numel()) * 4
            x = AttnMmaExtra(cu_seqlens=batch.cu_seqlens.data_ptr(), o_part=_ptr(o_part), ml_part=_ptr(ml_part),
                             n_segments=len(batch.segments), tokens_per_block=tpb, n_splits=splits,
                             seg_min_tokens=0, seg_max_tokens=big_from - 1)
            st = self._lib("attention_mma").spite_paged_attention_mma(
                C.byref(p), C.byref(b), C.byref(c), C.byref(x), n_small, self._stream())
            self._count("attention_mma", 1 + (splits > 1))
            _check(st, "paged_attention (tensor cores)")
            return
        st = self._lib("attention").spite_paged_attention(self._dt, C.byref(p), C.byref(b), C.byref(c),
                                                          self._stream())
        self._count("attention", 1)
        _check(st, "paged_attention")

    def _attention_decode(self, p, b, c, batch, n_small, tpb, seg_max, longest, num_heads, cache_settled):
        """Decoded tokens (and portions too short for the row kernels) on the TMA-fed decode kernel: as many
        key splits as fill the resident blocks once, partial results merged by the last block of a split set."""
        # 64 keys and 64 values of one kv head; keys that are the values, with a factor each, are one tile
        stage = (1 if c.key_scale else 2) * c.head_dim * 64 * 2
        tiles = -(-longest // 64) + 1
        base = n_small * c.num_kv_heads
        narrow = tpb * (num_heads // c.num_kv_heads) <= 8
        per_sm = max(1, min(4 if not c.key_scale else 3 if narrow else 2, (225 * 1024) // (3 * stage + 2048)))
        slots = per_sm * self.sm_count
        if base <= slots:
            splits = slots // base
        elif base >= 4 * slots:
            splits = 1
        else:
            splits = max(range(1, 5), key=lambda s: (base * s / slots) / -(-base * s // slots))
        splits = max(1, min(splits, tiles // 2, self.attention_max_splits))
        deep = 6 if per_sm == 1 or (c.key_scale and per_sm == 2) else 4 if c.key_scale else 3
        n_stages = max(2, min(deep, -(-tiles // splits)))
        partial = tickets = None
        if splits > 1:
            if base > self._tickets_n:
                raise KernelError(f"paged_attention: {base} (request block, kv head) pairs exceed the {self._tickets_n} tickets")
            partial = torch.empty((base * splits * 16 * (c.head_dim + 4),), dtype=torch.float32, device=self.device)
            self.attention_scratch_bytes = partial.numel() * 4
            tickets = self._tickets_of(torch.cuda.current_stream().cuda_stream)
        x = AttnDecodeExtra(cu_seqlens=batch.cu_seqlens.data_ptr(), partial=_ptr(partial), tickets=_ptr(tickets),
                            n_segments=len(batch.segments), tokens_per_block=tpb, n_splits=splits,
                            seg_min_tokens=0, seg_max_tokens=seg_max, cache_settled=int(bool(cache_settled)))
        st = self._lib("attention_decode").spite_paged_attention_decode(
            C.byref(p), C.byref(b), C.byref(c), C.byref(x), n_small, n_stages, self._stream())
        self._count("attention_decode", 1)
        _check(st, "paged_attention (decode)")

    # ------------------------------------------------------------------ attention through latents
    def latent_prepare(self, down, cq_out, batch, cache, *, q_rank, kv_rank, rotation, q_gain, kv_gain, eps,
                       num_gates=0, gates_out=None):
        self._t(down, torch.float32, "down"); self._t(cq_out, self.dtype, "cq_out")
        self._t(q_gain, torch.float32, "q_gain"); self._t(kv_gain, torch.float32, "kv_gain")
        inv_freq = self._t(rotation.inv_freq, torch.float32, "inv_freq")
        if q_gain.numel() != q_rank or kv_gain.numel() != kv_rank or tuple(cq_out.shape) != (down.shape[0], q_rank):
            raise KernelError("latent_prepare: shapes do not fit")
        if cache.kv.shape[0] != 1:
            raise KernelError("latent_prepare writes one row per position: the cache has one plane")
        if gates_out is not None and tuple(self._t(gates_out, torch.float32, "gates_out").shape) != (down.shape[0], num_gates):
            raise KernelError("latent_prepare: gates_out must be [tokens, gates]")
        p = LatentPrepareParams(down=down.data_ptr(), down_stride=down.shape[1], cq_out=cq_out.data_ptr(),
                                q_gain=q_gain.data_ptr(), kv_gain=kv_gain.data_ptr(), inv_freq=inv_freq.data_ptr(),
                                rot_amplitude=float(rotation.amplitude), eps=float(eps), q_rank=int(q_rank),
                                kv_rank=int(kv_rank), rot_dim=2 * inv_freq.numel(), num_gates=int(num_gates),
                                gates_out=_ptr(gates_out), write_cache=int(cache.write),
                                pairing={"neighbours": 0, "halves": 1}[rotation.pairing])
        b, c = self._step_tokens(batch, cache.group), self._paged(cache)
        st = self._lib("latent").spite_latent_prepare(self._dt, C.byref(p), C.byref(b), C.byref(c), self._stream())
        self._count("latent", 1)
        _check(st, "latent_prepare")

    def latent_queries(self, q, q_out, batch, *, num_heads, head_dim, kv_rank, rotation, rows_out, offsets_out,
                       sorted_out=None):
        self._t(q, self.dtype, "q"); self._t(q_out, self.dtype, "q_out")
        if sorted_out is not None and tuple(self._t(sorted_out, self.dtype, "sorted_out").shape) != (num_heads * q.shape[0], head_dim):
            raise KernelError("latent_queries: sorted_out must be [heads * tokens, head_dim]")
        self._t(rows_out, torch.int32, "rows_out"); self._t(offsets_out, torch.int32, "offsets_out")
        inv_freq = self._t(rotation.inv_freq, torch.float32, "inv_freq")
        M, rot = q.shape[0], 2 * inv_freq.numel()
        if q.shape[1] != num_heads * (head_dim + rot) or q_out.shape[0] != M or q_out.shape[1] % num_heads \
                or rows_out.numel() != num_heads * M or offsets_out.numel() != num_heads + 1:
            raise KernelError("latent_queries: shapes do not fit")
        p = LatentQueryParams(q=q.data_ptr(), q_out=q_out.data_ptr(), inv_freq=inv_freq.data_ptr(),
                              rot_amplitude=float(rotation.amplitude), num_heads=int(num_heads), head_dim=int(head_dim),
                              rot_dim=rot, kv_rank=int(kv_rank), row=q_out.shape[1] // num_heads,
                              positions=batch.positions.data_ptr(), n_tokens=M, rows_out=rows_out.data_ptr(),
                              offsets_out=offsets_out.data_ptr(), q_sorted_out=_ptr(sorted_out),
                              pairing={"neighbours": 0, "halves": 1}[rotation.pairing])
        st = self._lib("latent").spite_latent_queries(self._dt, C.byref(p), self._stream())
        self._count("latent", 1)
        _check(st, "latent_queries")

    # ------------------------------------------------------------------ recurrent mixers
    def mlstm_scan(self, proj, out, batch, state, *, heads, dim, vdim, gate_cap, q_scale, columns, i_bias, f_bias,
                   chunked=None):
        self._t(proj, torch.float32, "proj"); self._t(out, torch.float32, "out"); self._t(state, torch.float32, "state")
        self._t(i_bias, torch.float32, "i_bias"); self._t(f_bias, torch.float32, "f_bias")
        M = proj.shape[0]
        q_col, k_col, v_col, i_col, f_col = (int(c) for c in columns)
        if tuple(out.shape) != (M, heads * vdim) or state.dim() != 3 or state.shape[1] != heads \
                or state.shape[2] < self.mlstm_state_size(dim, vdim) or i_bias.numel() != heads or f_bias.numel() != heads:
            raise KernelError("mlstm_scan: shapes do not fit")
        if max(q_col + heads * dim, k_col + heads * dim, v_col + heads * vdim, i_col + heads, f_col + heads) > proj.shape[1]:
            raise KernelError("mlstm_scan: the columns lie outside the projection's rows")
        n_seg = batch.cu_seqlens.numel() - 1
        if chunked is None:
            # Prompts and their portions go 32 tokens at a time.  The float32 set keeps the walk token by token for
            # every step, so that its results do not depend on how a prompt was cut, to the last bit.
            chunked = self.dtype != torch.float32 and batch.max_seg_len >= 8
        p = MlstmParams(proj=proj.data_ptr(), stride=proj.shape[1], q_col=q_col, k_col=k_col, v_col=v_col, i_col=i_col,
                        f_col=f_col, i_bias=i_bias.data_ptr(), f_bias=f_bias.data_ptr(), out=out.data_ptr(),
                        state=state.data_ptr(), head_stride=state.shape[2], cu_seqlens=batch.cu_seqlens.data_ptr(),
                        slots=batch.slots.data_ptr(), n_segments=n_seg, heads=int(heads), dim=int(dim), vdim=int(vdim),
                        gate_cap=float(gate_cap), q_scale=float(q_scale), chunked=int(bool(chunked)))
        if chunked:
            # working memory for what the chunks need ahead of the state (scores, sums of the gates): a record for every
            # chunk and head; the segments' chunks are at most tokens / 32 + segments
            n_chunks = (M + 31) // 32 + n_seg
            scratch = torch.empty((n_chunks, heads, 1152), dtype=torch.float32, device=proj.device)
            st = self._lib("recurrent").spite_mlstm_scan_chunked(C.byref(p), C.c_void_p(scratch.data_ptr()), C.c_int(n_chunks), self._stream())
        else:
            st = self._lib("recurrent").spite_mlstm_scan(C.byref(p), self._stream())
        self._count("recurrent", 2 if chunked else 1)
        _check(st, "mlstm_scan")

    def delta_scan(self, x, out, batch, state, *, heads, kv_heads, dim, vdim, columns, a_log, dt_bias, q_scale,
                   unit_eps=1e-6, state_offset=0, split_rows=None):
        self._t(x, torch.float32, "x"); self._t(out, torch.float32, "out"); self._t(state, torch.float32, "state")
        self._t(a_log, torch.float32, "a_log"); self._t(dt_bias, torch.float32, "dt_bias")
        M = x.shape[0]
        q_col, k_col, v_col, b_col, a_col = (int(c) for c in columns)
        slot_stride = state[0].numel()
        if tuple(out.shape) != (M, heads * vdim) or a_log.numel() != heads or dt_bias.numel() != heads or heads % kv_heads \
                or state_offset < 0 or state_offset + heads * dim * vdim > slot_stride:
            raise KernelError("delta_scan: shapes do not fit")
        if max(q_col + kv_heads * dim, k_col + kv_heads * dim, v_col + heads * vdim, b_col + heads, a_col + heads) > x.shape[1]:
            raise KernelError("delta_scan: the columns lie outside the rows of x")
        # what a token brings besides q, k, v (unit-vector factors, beta, decay): filled by the first of the two kernels
        gates = torch.empty((M, 2 * kv_heads + 2 * heads), dtype=torch.float32, device=x.device)
        p = DeltaParams(x=x.data_ptr(), stride=x.shape[1], q_col=q_col, k_col=k_col, v_col=v_col, b_col=b_col, a_col=a_col,
                        a_log=a_log.data_ptr(), dt_bias=dt_bias.data_ptr(), out=out.data_ptr(),
                        state=state.data_ptr() + 4 * int(state_offset), slot_stride=slot_stride,
                        cu_seqlens=batch.cu_seqlens.data_ptr(), slots=batch.slots.data_ptr(),
                        n_segments=batch.cu_seqlens.numel() - 1, heads=int(heads), kv_heads=int(kv_heads), dim=int(dim),
                        vdim=int(vdim), q_scale=float(q_scale), unit_eps=float(unit_eps), gates=gates.data_ptr(), n_tokens=M)
        if split_rows is None:
            # A warp on eight value columns (whole sectors of the state per row) serves every step.  More lanes a column
            # and fewer columns a block was measured and is no faster: the walk's time is the length of its chain per token
            # (a barrier, the sums, the shuffles), not the multiply-adds (2,048 tokens of 16 heads of 128 x 128: 1.73 ms
            # against 2.05 ms; eight such prompts 3.48 against 3.98 ms).  One form for every step also keeps the float32
            # set's results independent of how a prompt was cut, to the last bit.
            split_rows = False
        st = self._lib("delta").spite_delta_scan(C.byref(p), C.c_int(int(bool(split_rows))), self._stream())
        self._count("delta", 2)
        _check(st, "delta_scan")

    def _scan(self, what, q, k, v, out, batch, state, *, heads, kv_heads, dim, vdim, state_offset, scalars=True):
        """The argument block that the scans share; q, k, v are (float32 tensor [M, *], first column)."""
        self._t(out, torch.float32, "out"); self._t(state, torch.float32, "state")
        M = out.shape[0]
        slot_stride = state[0].numel()
        if tuple(out.shape) != (M, heads * vdim) or heads % kv_heads or state_offset < 0 \
                or state_offset + heads * self.scan_state_size(dim, vdim) > slot_stride:
            raise KernelError(f"{what}: shapes do not fit")
        at = []
        for name, (t, column), width in (("q", q, kv_heads * dim), ("k", k, kv_heads * dim), ("v", v, heads * vdim)):
            self._t(t, torch.float32, name)
            at.append((self._columns(t, column, width, M, f"{what}: {name}"), t.shape[1]))
        scalars = torch.empty((M, heads, 4), dtype=torch.float32, device=out.device) if scalars else None
        p = ScanParams(q=at[0][0], k=at[1][0], v=at[2][0], q_stride=at[0][1], k_stride=at[1][1], v_stride=at[2][1],
                       w=None, w_stride=0, scalars=_ptr(scalars), skip=None, out=out.data_ptr(), out_stride=out.shape[1],
                       state=state.data_ptr() + 4 * int(state_offset), slot_stride=slot_stride,
                       cu_seqlens=batch.cu_seqlens.data_ptr(), slots=batch.slots.data_ptr(),
                       n_segments=batch.cu_seqlens.numel() - 1, n_tokens=M, heads=int(heads), kv_heads=int(kv_heads),
                       dim=int(dim), vdim=int(vdim))
        return p, scalars

    def state_space_scan(self, q, k, v, step, out, batch, state, *, heads, kv_heads, dim, vdim, a_log, dt_bias, skip,
                         state_offset=0):
        p, scalars = self._scan("state_space_scan", q, k, v, out, batch, state, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim,
                                state_offset=state_offset)
        for name, t in (("a_log", a_log), ("dt_bias", dt_bias), ("skip", skip)):
            if self._t(t, torch.float32, name).numel() != heads:
                raise KernelError(f"state_space_scan: {name} has one element per head")
        t, column = step
        self._t(t, torch.float32, "step")
        a = self._columns(t, column, heads, out.shape[0], "state_space_scan: step")
        p.skip = skip.data_ptr()
        st = self._lib("scan").spite_state_space_scan(C.byref(p), C.c_void_p(a), C.c_longlong(t.shape[1]),
                                                      C.c_void_p(a_log.data_ptr()), C.c_void_p(dt_bias.data_ptr()), self._stream())
        self._count("scan", 2)
        _check(st, "state_space_scan")

    def decay_scan(self, r, k, v, w, out, batch, state, *, heads, dim, vdim, w0, u, state_offset=0):
        p, scalars = self._scan("decay_scan", r, k, v, out, batch, state, heads=heads, kv_heads=heads, dim=dim, vdim=vdim,
                                state_offset=state_offset)
        self._t(w, torch.float32, "w")
        if tuple(w.shape) != (out.shape[0], heads * dim):
            raise KernelError("decay_scan: w must be [tokens, heads * dim]")
        for name, t in (("w0", w0), ("u", u)):
            if self._t(t, torch.float32, name).numel() != heads * dim:
                raise KernelError(f"decay_scan: {name} has one element per head and key channel")
        p.w, p.w_stride = w.data_ptr(), w.shape[1]
        st = self._lib("scan").spite_decay_scan(C.byref(p), C.c_void_p(w0.data_ptr()), C.c_void_p(u.data_ptr()), self._stream())
        self._count("scan", 2)
        _check(st, "decay_scan")

    def gated_linear_scan(self, q, k, v, a, w, out, batch, state, *, heads, dim, vdim, a2, a2_bias, tau, q_scale, state_offset=0):
        p, _ = self._scan("gated_linear_scan", q, k, v, out, batch, state, heads=heads, kv_heads=heads, dim=dim, vdim=vdim,
                          state_offset=state_offset, scalars=False)
        self._t(w, torch.float32, "w"); self._t(a2, torch.float32, "a2")
        n, rank = heads * dim, a2.shape[0]
        if tuple(w.shape) != (out.shape[0], n) or tuple(a2.shape) != (rank, n) or self._t(a2_bias, torch.float32, "a2_bias").numel() != n:
            raise KernelError("gated_linear_scan: w is [tokens, heads * dim], a2 [rank, heads * dim], its bias [heads * dim]")
        t, column = a
        self._t(t, torch.float32, "a")
        at = self._columns(t, column, rank, out.shape[0], "gated_linear_scan: a")
        p.w, p.w_stride, p.out_scale = w.data_ptr(), n, float(q_scale)
        st = self._lib("scan").spite_gated_linear_scan(C.byref(p), C.c_void_p(at), C.c_longlong(t.shape[1]), C.c_void_p(a2.data_ptr()),
                                                       C.c_void_p(a2_bias.data_ptr()), int(rank), C.c_float(tau), self._stream())
        self._count("scan", 2)
        _check(st, "gated_linear_scan")

    # ------------------------------------------------------------------ mixture of experts
    def moe_identity(self, x, routing, first_identity, out, *, accumulate=True):
        self._t(x, self.dtype, "x"); self._t(out, torch.float32, "out")
        M, d = x.shape
        top_k = routing.expert_ids.shape[0]
        if tuple(out.shape) != (M, d) or routing.expert_ids.shape[1] != M or tuple(routing.weights.shape) != (top_k, M):
            raise KernelError("moe_identity: shapes do not fit")
        st = self._lib("moe").spite_moe_identity(
            self._dt, C.c_void_p(x.data_ptr()), C.c_void_p(routing.expert_ids.data_ptr()), C.c_void_p(routing.weights.data_ptr()),
            M, d, top_k, int(first_identity), C.c_void_p(out.data_ptr()), int(bool(accumulate)), self._stream())
        self._count("moe", 1)
        _check(st, "moe_identity")

    def moe_route(self, x, w_router, top_k, want_logits=False, scoring="sigmoid", choice_bias=None, logit_bias=None) -> Routing:
        if scoring not in ("sigmoid", "softmax_renorm", "softmax_biased"):
            raise KernelError(f"moe_route: unknown scoring {scoring!r}")
        if (scoring == "softmax_biased") != (choice_bias is not None):
            raise KernelError("moe_route: `choice_bias` goes with the scoring 'softmax_biased'")
        if choice_bias is not None and self._t(choice_bias, torch.float32, "choice_bias").numel() != w_router.shape[0]:
            raise KernelError("moe_route: one choice bias per expert")
        if logit_bias is not None and self._t(logit_bias, torch.float32, "logit_bias").numel() != w_router.shape[0]:
            raise KernelError("moe_route: one logit bias per expert")
        self._t(x, self.dtype, "x"); self._t(w_router, torch.float32, "w_router")
        M, d = x.shape
        E = w_router.shape[0]
        dev = x.device
        ids = torch.empty((top_k, M), dtype=torch.int32, device=dev)
        wts = torch.empty((top_k, M), dtype=torch.float32, device=dev)
        offsets = torch.empty((top_k, E + 1), dtype=torch.int32, device=dev)
        rows = torch.empty((top_k, M), dtype=torch.int32, device=dev)
        logits = torch.empty((M, E), dtype=torch.float32, device=dev)
        renorm = {"sigmoid": 0, "softmax_renorm": 1, "softmax_biased": 2}[scoring]
        sorted_w = torch.empty((top_k, M), dtype=torch.float32, device=dev) if renorm else None
        st = self._lib("moe").spite_moe_route(
            self._dt, C.c_void_p(x.data_ptr()), C.c_void_p(w_router.data_ptr()), M, d, E, top_k,
            C.c_void_p(ids.data_ptr()), C.c_void_p(wts.data_ptr()), C.c_void_p(_ptr(logits)),
            C.c_void_p(offsets.data_ptr()), C.c_void_p(rows.data_ptr()), int(renorm), C.c_void_p(_ptr(sorted_w)),
            C.c_void_p(_ptr(choice_bias)), C.c_void_p(_ptr(logit_bias)), self._stream())
        self._count("moe", 2 if M <= 64 else 3)
        _check(st, "moe_route")
        return Routing(ids, wts, offsets, rows, logits if want_logits else None, sorted_w)

    # ------------------------------------------------------------------ sampling
    def argmax(self, logits):
        self._t(logits, torch.float32, "logits")
        R, V = logits.shape
        out = torch.empty(R, dtype=torch.int32, device=logits.device)
        st = self._lib("sampling").spite_argmax(C.c_void_p(logits.data_ptr()), R, V,
                                                C.c_void_p(out.data_ptr()), self._stream())
        self._count("sampling", 1)
        _check(st, "argmax")
        return out

    def sample(self, logits, *, temperature, top_k=None, top_p=None, min_p=None, repetition_penalty=None,
               context=None, context_offsets=None, rng_state):
        self._t(logits, torch.float32, "logits"); self._t(temperature, torch.float32, "temperature")
        self._t(rng_state, torch.int64, "rng_state")
        R, V = logits.shape
        work = torch.empty_like(logits)
        out = torch.empty(R, dtype=torch.int32, device=logits.device)
        p = SampleParams(logits=logits.data_ptr(), work=work.data_ptr(), temperature=temperature.data_ptr(),
                         top_k=_ptr(top_k), top_p=_ptr(top_p), min_p=_ptr(min_p),
                         repetition_penalty=_ptr(repetition_penalty), context=_ptr(context),
                         context_offsets=_ptr(context_offsets), rng_state=rng_state.data_ptr(),
                         out_tokens=out.data_ptr(), vocab=V)
        st = self._lib("sampling").spite_sample(C.byref(p), R, self._stream())
        self._count("sampling", 1)
        _check(st, "sample")
        return out
