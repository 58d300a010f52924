#!/usr/bin/env bash
# Builds the sm_100a libraries (CUDA kernels + C ABI) in tree, one object per source, in parallel:
#   lib/libmllm_b200.so     quantized linears, the quantized decoder, tensor parallelism   (include/mllmb200.h)
#   lib/libmllm_b200_lm.so  bf16 language-model engine                                     (include/mllmb200_lm.h)
# Usage: build.sh [all|core|lm].  Objects whose sources have not changed are kept.
set -euo pipefail
HERE="$(cd "$(dirname "${BASH_SOURCE[0]}")" && pwd)"
NVCC="${NVCC:-/usr/local/cuda/bin/nvcc}"
[ -x "$NVCC" ] || NVCC=nvcc
WHAT="${1:-all}"
OUT="$HERE/lib"
OBJ="$HERE/build"
CORE=(host_pack.cpp c_api.cu device_status.cu repack.cu act_quant.cu gemv.cu gemv_stream.cu gemm_stream.cu gemm_simt.cu gemm_tc.cu
      gemm_tcf16.cu decoder_kernels.cu decoder_attn.cu decoder_sample.cu decoder.cu decoder_batch.cu decoder_persistent.cu conv3d.cu
      host_pack_a16.cpp w4a16.cu c_api_a16.cu tp.cu)
[ -f "$HERE/csrc/no_alloc.cu" ] && CORE+=(no_alloc.cu)
LM=(lm/lm_engine.cu lm/lm_linear.cu lm/lm_norm.cu lm/lm_attn.cu lm/lm_latent.cu lm/lm_moe.cu lm/lm_retention.cu device_status.cu decoder_sample.cu)
FLAGS=(-std=c++17 -O3 -gencode arch=compute_100a,code=sm_100a -lineinfo -rdc=true -Xcompiler -fPIC,-fvisibility=hidden,-O3)
[ -n "${PTXAS_V:-}" ] && FLAGS+=(-Xptxas -v)

# what an object depends on: every header, its own source, the flags
HEADERS="$(cat "$HERE"/csrc/*.h "$HERE"/csrc/*.cuh "$HERE"/csrc/*.inc "$HERE"/csrc/lm/*.h "$HERE"/csrc/lm/*.cuh "$HERE"/../include/*.h | sha256sum)"
compile() {
  local src="$1" obj stamp
  obj="$OBJ/$(echo "$src" | tr '/.' '__').o"
  stamp="$(echo "$HEADERS ${FLAGS[*]} $(sha256sum <"$HERE/csrc/$src")" | sha256sum)"
  [ -f "$obj" ] && [ "$(cat "$obj.stamp" 2>/dev/null)" = "$stamp" ] && return 0
  "$NVCC" "${FLAGS[@]}" -c "$HERE/csrc/$src" -o "$obj.$$.o" && mv "$obj.$$.o" "$obj" || return 1
  echo "$stamp" >"$obj.stamp"
}
link() {
  local lib="$1"
  shift
  local objs=()
  for s in "$@"; do objs+=("$OBJ/$(echo "$s" | tr '/.' '__').o"); done
  "$NVCC" -gencode arch=compute_100a,code=sm_100a -shared -o "$OUT/$lib.$$" "${objs[@]}" -ldl
  mv "$OUT/$lib.$$" "$OUT/$lib"
  echo "built $OUT/$lib"
}

stamp_of() { (cd "$HERE/csrc" && echo "$HEADERS ${FLAGS[*]} $(sha256sum "$@")" | sha256sum); }
current() {  # library, its sources: built from these?
  local lib="$1"
  shift
  [ -f "$OUT/$lib" ] && [ "$(cat "$OUT/.$lib.stamp" 2>/dev/null)" = "$(stamp_of "$@")" ]
}
todo() {
  SRC=()
  NEED_CORE=0
  NEED_LM=0
  case "$WHAT" in all | core) current libmllm_b200.so "${CORE[@]}" || { NEED_CORE=1; SRC+=("${CORE[@]}"); } ;; esac
  case "$WHAT" in all | lm) current libmllm_b200_lm.so "${LM[@]}" || { NEED_LM=1; SRC+=("${LM[@]}"); } ;; esac
  [ ${#SRC[@]} -gt 0 ]
}

case "$WHAT" in all | core | lm) ;; *) echo "usage: build.sh [all|core|lm]" >&2; exit 2 ;; esac
todo || exit 0
mkdir -p "$OUT" "$OBJ"
exec 9>"$OBJ/.lock"  # one build at a time
flock 9
todo || exit 0
JOBS="$(nproc)"
rm -f "$OBJ/.failed"
declare -A started=()
for s in "${SRC[@]}"; do
  [ -n "${started[$s]:-}" ] && continue
  started[$s]=1
  while [ "$(jobs -rp | wc -l)" -ge "$JOBS" ]; do wait -n || true; done
  { compile "$s" || touch "$OBJ/.failed"; } 9>&- &
done
wait
[ ! -e "$OBJ/.failed" ] || { echo "build.sh: a source did not compile" >&2; exit 1; }
finish() {
  link "$@"
  local lib="$1"
  shift
  stamp_of "$@" >"$OUT/.$lib.stamp"
}
[ "$NEED_CORE" = 0 ] || finish libmllm_b200.so "${CORE[@]}"
[ "$NEED_LM" = 0 ] || finish libmllm_b200_lm.so "${LM[@]}"
