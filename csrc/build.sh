#!/usr/bin/env bash
# Builds the kernel library (sm_100a only) in-tree under distributed_llm_pipeline_b200/ops/:
#   build.sh          libdlp_b200.so         everything
#   build.sh layers   libdlp_b200_layers.so  what a layer-list model runs (a fresh checkout compiles this part first, in a fraction of the time)
set -euo pipefail
HERE="$(cd "$(dirname "$0")" && pwd)"
PART="${1:-all}"
OUT="$HERE/../distributed_llm_pipeline_b200/ops"
NVCC="${NVCC:-/usr/local/cuda/bin/nvcc}"
FLAGS=(-gencode arch=compute_100a,code=sm_100a -O3 -lineinfo -std=c++17 -Xcompiler -fPIC -Xptxas -v)
case "$PART" in
  all) OBJ="$HERE/build"; LIB="$OUT/libdlp_b200.so"; SRC=("$HERE"/*.cu) ;;
  layers) OBJ="$HERE/build/layers"; LIB="$OUT/libdlp_b200_layers.so"; FLAGS+=(-DDLP_LAYERS_ONLY)
          SRC=("$HERE"/layers_*.cu "$HERE"/capi_layers.cu "$HERE"/capi_core.cu "$HERE"/elementwise.cu "$HERE"/gemm_tcgen05.cu "$HERE"/moe.cu) ;;
  *) echo "build.sh: unknown part '$PART'" >&2; exit 2 ;;
esac
mkdir -p "$OBJ" "$OUT"
pids=()
objs=()
for f in "${SRC[@]}"; do
  b="$(basename "$f" .cu)"
  objs+=("$OBJ/$b.o")
  MATH=(--use_fast_math)
  case "$b" in layers_*_tc) ;; layers_*) MATH=() ;; esac        # exact divisions, square roots and exponentials where a layer is specified in 32 bits
  if [[ ! -f "$OBJ/$b.o" || "$f" -nt "$OBJ/$b.o" || -n "$(find "$HERE" -maxdepth 1 -name '*.cuh' -newer "$OBJ/$b.o" -print -quit)" || "$HERE/../include/dlp_b200.h" -nt "$OBJ/$b.o" ]]; then
    ( "$NVCC" "${FLAGS[@]}" ${MATH[@]+"${MATH[@]}"} -c "$f" -o "$OBJ/$b.o.tmp" > "$OBJ/$b.log" 2>&1 && mv "$OBJ/$b.o.tmp" "$OBJ/$b.o" || { cat "$OBJ/$b.log"; exit 1; } ) &
    pids+=($!)
  fi
done
for p in "${pids[@]:-}"; do [[ -n "$p" ]] && wait "$p"; done
"$NVCC" -gencode arch=compute_100a,code=sm_100a -shared -o "$LIB.tmp$$" "${objs[@]}" -lcudart_static -lpthread -ldl -lrt
mv "$LIB.tmp$$" "$LIB"
echo "built $LIB"
